"""Latent attention (keys and values of all heads expand from one cached vector per token) over the paged cache.

A cached row is ``[c | kr]``: the normalised latent (``rank`` wide) and one rotated key part (``rot`` wide) that all heads share.
With per-head expansions ``k = [W_uk c | kr]`` and ``v = W_uv c`` the same attention has two forms:

* absorbed: queries are moved into latent space (``W_uk^T q``), every head attends over the cached rows as they are, and the
  attended latents are expanded to values afterwards. The cache is read once for all heads - decode, and portions that are
  short against the context they see;
* expanded: the keys and values of the visible context are formed by one GEMM and attended per head on the tcgen05 kernel -
  long portions, where the narrower heads cost a fraction of the arithmetic.

Both take a sliding window, sinks and the sigmoid output gate. ``*_ref`` functions are the fp32 restatements CPU tensors run.
"""
from __future__ import annotations

import numpy as np
import torch

from . import native
from .core import CLUSTER_SPLITS, PAGE, _sm_count, _tma_rows, linear
from .native import F, I, L, P, check, lib, ptr, status_word, stream_ptr

native.register("eredu_latent_prepare", I, [P] * 8 + [I] * 6 + [F, P])
native.register("eredu_rotate_heads", I, [P] * 3 + [I] * 6 + [P])
native.register("eredu_gather_rows", I, [P] * 3 + [I] * 3 + [P])
native.register("eredu_head_linear", I, [P] * 8 + [I] * 4 + [L] * 5 + [I] * 3 + [P])
native.register("eredu_latent_attn", I, [P] * 7 + [I] * 10 + [F, P, P])
native.register("eredu_attn_prefill_rows", I, [P] * 8 + [I] * 9 + [L] * 4 + [F, P, P])

MAX_RANK, MAX_ROW = 512, 640   # widest latent and cached row of the tensor-core form of absorbed attention
MAX_SIMT_RANK = 1024      # of its CUDA-core form


def _rotate(x, positions, inv_freq):
    """x [M, heads, 2 len(inv_freq)] fp32: pairs (i, i + half) turned by position * inv_freq[i]."""
    a = positions.float()[:, None] * inv_freq.float()[None, :]
    cos, sin = a.cos()[:, None, :], a.sin()[:, None, :]
    u, v = x.chunk(2, -1)
    return torch.cat((u * cos - v * sin, v * cos + u * sin), -1)


# ---------------------------------------------------------------------------------------------- preparation
def latent_prepare_ref(proj, q_rank, rank, rot, q_norm_w, kv_norm_w, eps, positions, slots, inv_freq, cache):
    def rms(t, w):
        return t * torch.rsqrt(t.square().mean(-1, keepdim=True) + eps) * w.float()

    x = proj.float()
    c = rms(x[:, q_rank:q_rank + rank], kv_norm_w)
    kr = _rotate(x[:, None, q_rank + rank:q_rank + rank + rot], positions, inv_freq)[:, 0]
    ok = slots >= 0
    cache.view(-1, rank + rot)[slots[ok]] = torch.cat((c, kr), -1)[ok].to(cache.dtype)
    return rms(x[:, :q_rank], q_norm_w).to(proj.dtype)


def latent_prepare(proj, q_rank, rank, rot, q_norm_w, kv_norm_w, eps, positions, slots, inv_freq, cache):
    """``proj`` [M, >= q_rank + rank + rot] = [query latent | latent | key part]: RMSNorm of both latents, rotation of the key part by
    the token's position, ``[latent | key part]`` stored as the token's row of ``cache`` [pages, 1, 16, rank + rot] (``slots``:
    negative = not stored). Returns the normalised query latent [M, q_rank]."""
    if not proj.is_cuda:
        return latent_prepare_ref(proj, q_rank, rank, rot, q_norm_w, kv_norm_w, eps, positions, slots, inv_freq, cache)
    assert positions.dtype == torch.int32 and slots.dtype == torch.int64 and inv_freq.dtype == torch.float32
    assert proj.stride(1) == 1 and cache.is_contiguous() and cache.dtype == proj.dtype and cache.shape[1:] == (1, PAGE, rank + rot)
    M = proj.shape[0]
    cq = torch.empty((M, q_rank), dtype=proj.dtype, device=proj.device)
    code = lib().eredu_latent_prepare(ptr(proj), ptr(cq), ptr(cache), ptr(positions), ptr(slots), ptr(inv_freq), ptr(q_norm_w),
                                      ptr(kv_norm_w), M, proj.stride(0), q_rank, rank, rot, 1 if proj.dtype == torch.float32 else 0,
                                      eps, stream_ptr(proj.device))
    check(code, "eredu_latent_prepare")
    return cq


# ---------------------------------------------------------------------------------------------- attention
def latent_attention_ref(q, cache, batch, uk, uv, gate, sinks, inv_freq, heads, dim, rot, scale, window):
    M, rank = q.shape[0], uk.shape[1]
    x = q.float().view(M, heads, dim + rot)
    q_abs = torch.einsum("mhd,hrd->mhr", x[..., :dim], uk.float())
    q_rot = _rotate(x[..., dim:], batch.positions, inv_freq)
    bounds = batch.cu_q.tolist() if batch.is_prefill else [i * batch.q_per_seq for i in range(batch.block_table.shape[0] + 1)]
    out = torch.zeros((M, heads, uv.shape[1]), dtype=torch.float32, device=q.device)
    for b, kv_len in enumerate(batch.seq_lens.tolist()):
        r0, r1 = bounds[b], bounds[b + 1]
        if r1 <= r0:
            continue
        n_pages = (kv_len + PAGE - 1) // PAGE
        ctx = cache[batch.block_table[b, :n_pages].long(), 0].reshape(-1, rank + rot)[:kv_len].float()
        s = (torch.einsum("qhr,tr->hqt", q_abs[r0:r1], ctx[:, :rank]) + torch.einsum("qhr,tr->hqt", q_rot[r0:r1], ctx[:, rank:])) * scale
        qpos = torch.arange(kv_len - (r1 - r0), kv_len, device=q.device)[:, None]
        kpos = torch.arange(kv_len, device=q.device)[None, :]
        hidden = (kpos > qpos) | ((kpos <= qpos - window) if window else (kpos < 0))
        s = s.masked_fill(hidden, float("-inf"))
        if sinks is not None:
            s = torch.cat((s, sinks.float()[:, None, None].expand(-1, r1 - r0, 1)), -1)
        p = torch.softmax(s, -1)[..., :kv_len]
        out[r0:r1] = torch.einsum("qhr,hvr->qhv", torch.einsum("hqt,tr->qhr", p, ctx[:, :rank]), uv.float())
    out = out.reshape(M, -1)
    if gate is not None:
        out = out * torch.sigmoid(gate.float())
    return out.to(q.dtype)


def head_linear(x, w, out, gate=None, in_rows=None, out_rows=None, rot=0, positions=None, inv_freq=None):
    """Per-head matrices: ``out[m, h, :N] = w[h] x[m, h, :K]`` with w [H, N, K]; x and out are [rows, H, *] views whose last axis is
    contiguous. ``gate`` [rows, H * N] (any row pitch): the result is multiplied by its sigmoid. ``in_rows`` / ``out_rows``: row m is
    read from / stored to (and gated by) that row instead. ``rot``: the ``rot`` entries of x behind the first K are turned by
    ``positions`` (rows as x) and stored behind the first N of the output."""
    H, N, K = w.shape
    M = in_rows.shape[0] if in_rows is not None else (out_rows.shape[0] if out_rows is not None else x.shape[0])
    assert x.stride(2) == 1 and out.stride(2) == 1 and w.is_contiguous() and x.dtype == w.dtype == out.dtype
    fp32 = x.dtype == torch.float32
    tc = not fp32 and all(v % 8 == 0 for v in (N, K, x.stride(0), x.stride(1), out.stride(0), out.stride(1))) \
        and x.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0 and out.data_ptr() % 4 == 0
    if gate is not None:
        assert gate.stride(1) == 1 and gate.dtype == x.dtype
        tc = tc and gate.stride(0) % 2 == 0 and gate.data_ptr() % 4 == 0
    code = lib().eredu_head_linear(ptr(x), ptr(w), ptr(out), ptr(gate), ptr(in_rows), ptr(out_rows), ptr(positions) if rot else None,
                                   ptr(inv_freq) if rot else None, M, H, N, K, x.stride(0), x.stride(1), out.stride(0), out.stride(1),
                                   gate.stride(0) if gate is not None else 0, rot, 1 if fp32 else 0, 1 if tc else 0, stream_ptr(x.device))
    check(code, "eredu_head_linear")
    return out


class _Portions:
    """How the sequences of one prompt batch are served under one window: ``expanded`` and ``absorbed`` are indices into the batch,
    the tensors are what the kernels read. Made once per batch and geometry."""

    def __init__(self, batch, portions, expanded, absorbed, window, device):
        def put(a, dt):
            t = torch.from_numpy(np.ascontiguousarray(a)).to(dt)
            return t.pin_memory().to(device, non_blocking=True)

        start = np.cumsum([0] + [n for _, n in portions])
        self.expanded, self.absorbed = expanded, absorbed
        if expanded:
            first = [max(0, portions[b][0] - window + 1) if window else 0 for b in expanded]      # oldest visible position
            length = [sum(portions[b]) - f for b, f in zip(expanded, first)]
            self.rows = int(sum(length))                                                          # context rows of all of them
            seq = np.repeat(np.asarray(expanded), length)
            pos = np.concatenate([np.arange(f, f + n) for f, n in zip(first, length)])
            # (query row 0, queries, context row 0, context rows) per sequence
            self.table = put(np.asarray([[start[b], portions[b][1], c, n] for b, c, n in
                                         zip(expanded, np.cumsum([0] + length[:-1]), length)], dtype=np.int32), torch.int32)
            self.max_q = max(portions[b][1] for b in expanded)
            seq_t, pos_t = put(seq, torch.int64), put(pos, torch.int64)
            self.slots = batch.block_table.long()[seq_t, pos_t // PAGE] * PAGE + pos_t % PAGE     # cache row of every context row
        if absorbed:
            whole = len(absorbed) == len(portions)
            idx = put(np.asarray(absorbed), torch.int64)
            n = [portions[b][1] for b in absorbed]
            self.rows_of = None if whole else put(np.concatenate([np.arange(start[b], start[b + 1]) for b in absorbed]), torch.int32)
            self.block_table = batch.block_table if whole else batch.block_table[idx].contiguous()
            self.seq_lens = batch.seq_lens if whole else batch.seq_lens[idx].contiguous()
            self.cu = batch.cu_q if whole else put(np.cumsum([0] + n), torch.int32)
            self.n, self.max_n = int(sum(n)), max(n)
            self.seen = max(min(sum(portions[b]), portions[b][1] + window - 1 if window else 1 << 30) for b in absorbed)


# The absorbed form runs on mma.sync tiles, the expanded one on tcgen05: arithmetic of the former counts this many times.
ABSORBED_COST = 4


def _plan(batch, heads_cost, window, dims_ok, device):
    """Splits a prompt batch by arithmetic per head: expanding the context costs its length, absorbing costs the queries."""
    key = (heads_cost, window, dims_ok)
    plans = batch.__dict__.setdefault("_latent_plans", {})
    if key not in plans:
        rank, dim, rot, vdim = heads_cost
        portions, expanded, absorbed = batch.host_portions(), [], []
        for b, (at, n) in enumerate(portions):
            if n <= 0:
                continue
            ctx = min(at, window - 1) + n if window else at + n
            pairs = n * (min(window, ctx) if window else at + n / 2)
            expand = ctx * rank * (dim + vdim) + pairs * (dim + rot + vdim)
            absorb = (n * rank * (dim + vdim) + pairs * (2 * rank + rot)) * ABSORBED_COST
            (expanded if dims_ok and n >= 8 and expand < absorb else absorbed).append(b)
        plans[key] = _Portions(batch, portions, expanded, absorbed, window, device)
    return plans[key]


def latent_tile(rows: int, rank: int, rot: int) -> tuple:
    """(rows of a CTA, CTAs an SM holds) of the absorbed form for sequences of ``rows`` (token, head) pairs."""
    tile = 64 if rows > 32 else (32 if rows > 16 else 16)
    return tile, 2 if tile < 64 and rank <= 256 and rank + rot <= 320 else 1


def latent_splits(batch: int, row_tiles: int, seen: int, ctas: int) -> int:
    """Split-KV factor of the absorbed form: about as many CTAs as fit at once (``ctas``), at least two steps of 64 keys per split,
    one cluster at most."""
    steps = max(1, -(-seen // 32))
    return max(1, min(CLUSTER_SPLITS, ctas // max(1, batch * row_tiles), steps // 4 or 1))


def _absorbed(q, cache, uk, uv, gate, sinks, inv_freq, positions, heads, dim, rot, scale, window, block_table, seq_lens, cu, q_per_seq,
              max_n, seen, rows, out):
    """Absorbed attention of the query rows ``rows`` (None: all) into ``out`` [M, heads, vdim]."""
    dev, rank = q.device, uk.shape[1]
    M = q.shape[0] if rows is None else rows.shape[0]
    q_abs = torch.empty((M, heads, rank + rot), dtype=q.dtype, device=dev)
    head_linear(q.view(-1, heads, dim + rot), uk, q_abs, in_rows=rows, rot=rot, positions=positions, inv_freq=inv_freq)
    lat = torch.empty((M, heads, rank), dtype=q.dtype, device=dev)
    B = seq_lens.shape[0]
    tc = q.dtype == torch.bfloat16 and rank % 8 == 0 and rot % 8 == 0 and rank <= MAX_RANK and rank + rot <= MAX_ROW
    if tc:
        tile, per_sm = latent_tile(heads * max_n, rank, rot)
        splits = latent_splits(B, -(-heads * max_n // tile), seen, per_sm * _sm_count(dev))
        code = lib().eredu_latent_attn(ptr(q_abs), ptr(cache), ptr(lat), ptr(block_table), ptr(seq_lens), ptr(cu), ptr(sinks), B, q_per_seq,
                                       max_n, block_table.stride(0), heads, rank, rot, tile, splits, window, scale, ptr(status_word(dev)),
                                       stream_ptr(dev))
        check(code, "eredu_latent_attn")
    else:
        assert rank <= MAX_SIMT_RANK
        code = lib().eredu_attn_simt(ptr(q_abs), ptr(cache), ptr(cache), ptr(lat), ptr(block_table), ptr(seq_lens), ptr(cu), ptr(sinks), B,
                                     q_per_seq, max_n, block_table.stride(0), heads, 1, rank + rot, rank, rank + rot, window, 0,
                                     1 if q.dtype == torch.float32 else 0, scale, stream_ptr(dev))
        check(code, "eredu_attn_simt")
    head_linear(lat, uv, out, gate=gate, out_rows=rows)


def _expanded(q, cache, kv_up, gate, sinks, inv_freq, positions, heads, dim, rot, vdim, scale, window, plan, out):
    """Attention of the sequences of ``plan.expanded`` over keys and values expanded from their visible context."""
    dev, rank = q.device, kv_up.shape[1]
    M = q.shape[0]
    q = q.clone() if plan.absorbed else q              # the absorbed rows are rotated where they are used
    code = lib().eredu_rotate_heads(ptr(q), ptr(positions), ptr(inv_freq), M, q.stride(0), heads, dim + rot, dim, rot, stream_ptr(dev))
    check(code, "eredu_rotate_heads")
    ctx = torch.empty((plan.rows, rank + rot), dtype=q.dtype, device=dev)
    code = lib().eredu_gather_rows(ptr(cache), ptr(plan.slots), ptr(ctx), plan.rows, rank + rot, 2, stream_ptr(dev))
    check(code, "eredu_gather_rows")
    kv = linear(ctx[:, :rank], kv_up)                                    # [rows, H dim | H vdim]
    keys = heads * dim
    code = lib().eredu_attn_prefill_rows(ptr(q), ptr(kv), kv.data_ptr() + keys * 2, ctx.data_ptr() + rank * 2, ptr(gate), ptr(sinks),
                                         ptr(out), ptr(plan.table), plan.table.shape[0], M, plan.rows, plan.max_q, heads, dim, rot,
                                         vdim, window, q.stride(0), kv.stride(0), rank + rot, gate.stride(0) if gate is not None else 0,
                                         scale, ptr(status_word(dev)), stream_ptr(dev))
    check(code, "eredu_attn_prefill_rows")


def latent_attention(q, cache, batch, uk, uv, kv_up, gate, sinks, inv_freq, heads, dim, rot, scale, window=0):
    """``q`` [M, heads * (dim + rot)]: queries before rotation, head by head [unrotated | rotated]. ``cache`` [pages, 1, 16, rank + rot]
    holds the batch's rows already (:func:`latent_prepare`). ``uk`` [heads, rank, dim] (the transposed key expansion), ``uv``
    [heads, vdim, rank], ``kv_up`` [heads * (dim + vdim), rank] both expansions stacked. ``gate`` [M, heads * vdim]: sigmoid output
    gate before its activation, or None; ``sinks`` fp32 [heads] or None. Returns [M, heads * vdim]."""
    if not q.is_cuda:
        return latent_attention_ref(q, cache, batch, uk, uv, gate, sinks, inv_freq, heads, dim, rot, scale, window)
    M, rank, vdim = q.shape[0], uk.shape[1], uv.shape[1]
    assert q.is_contiguous() and cache.is_contiguous() and cache.dtype == q.dtype and cache.shape[1:] == (1, PAGE, rank + rot)
    assert sinks is None or (sinks.dtype == torch.float32 and sinks.is_contiguous())
    out = torch.empty((M, heads, vdim), dtype=q.dtype, device=q.device)
    if M == 0:
        return out.view(M, -1)
    common = (q, cache, uk, uv, gate, sinks, inv_freq, batch.positions, heads, dim, rot, scale, window)
    if not batch.is_prefill:
        seen = min(batch.max_kv_len or (1 << 30), window) if window else (batch.max_kv_len or 1 << 30)
        _absorbed(*common, batch.block_table, batch.seq_lens, None, batch.q_per_seq, batch.q_per_seq, seen, None, out)
        return out.view(M, -1)
    dims_ok = (q.dtype == torch.bfloat16 and all(v % 8 == 0 for v in (dim, rot, vdim, rank)) and 0 < dim <= 128 and 0 < rot <= 64
               and vdim <= 128 and (gate is None or _tma_rows(gate)))
    plan = _plan(batch, (rank, dim, rot, vdim), window, dims_ok, q.device)
    if plan.absorbed:
        _absorbed(*common, plan.block_table, plan.seq_lens, plan.cu, 0, plan.max_n, plan.seen, plan.rows_of, out)
    if plan.expanded:
        _expanded(q, cache, kv_up, gate, sinks, inv_freq, batch.positions, heads, dim, rot, vdim, scale, window, plan, out)
    return out.view(M, -1)
