"""Causal short convolutions with recurrent state: the gated operator of LFM2's "conv" layers, and the convolutions of projections
in front of attention and selective scans (:func:`conv_project`).

``proj = in_proj(x) = [B | C | X]``; ``bx = B * X``; ``y[t] = sum_j w[:, j] * bx[t - (L-1) + j]`` (depthwise, causal);
``out = C * (y + bias)`` (eredu/src/backend/mlx/architectures/lfm2/model.rs:899-914; the rolling cache of the last
L-1 inputs is ``CausalConv1dCache``). The state pool ``[pages, L-1, C]`` is indexed by each sequence's first KV page
(column 0 of the block table), so chunked prefill, decode and mixed batches share one code path and a captured
decode graph needs no host-side indices.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from . import native
from .native import I, P, check, lib, ptr, stream_ptr
from .pooling import PAGE, pool_block_ref
from .recurrent import _sequences

native.register("eredu_short_conv", I, [P, I, P, P, P, P, I, P, I, P, P, P, I, I, I, I, I, I, P])


def short_conv_ref(proj, w, bias, state, block_table, cu_q, q_per_seq, positions, slots, mode=0, x_off=0):
    """PyTorch reference (any device, fp32 maths, bx and the state rounded to the state's dtype like the kernel).
    mode 0: gated LFM2 form over proj = [B | C | X]; mode 1: silu(conv(proj[:, x_off : x_off + C]))."""
    M = proj.shape[0]
    C = w.shape[0]
    L = w.shape[1]
    out = torch.zeros((M, C), dtype=proj.dtype, device=proj.device)
    B = block_table.shape[0]
    bounds = cu_q.tolist() if cu_q is not None else [i * q_per_seq for i in range(B + 1)]
    wf = w.float()
    for b in range(B):
        r0, r1 = bounds[b], bounds[b + 1]
        if r1 <= r0 or int(slots[r0]) < 0:
            continue
        page = int(block_table[b, 0])
        pos0 = int(positions[r0])
        pj = proj[r0:r1].float()
        bx = (pj[:, x_off:x_off + C] if mode == 1 else (pj[:, :C] * pj[:, 2 * C:3 * C])).to(state.dtype).float()
        hist = state[page].float().clone()                         # [L-1, C]: positions pos0-(L-1) .. pos0-1
        for j in range(L - 1):
            if pos0 - (L - 1) + j < 0:
                hist[j] = 0
        full = torch.cat((hist, bx), 0)                            # [L-1+n, C]
        n = r1 - r0
        y = torch.zeros((n, C), dtype=torch.float32, device=proj.device)
        for j in range(L):
            y += wf[:, j][None, :] * full[j:j + n]
        if bias is not None:
            y += bias.float()[None, :]
        out[r0:r1] = (torch.nn.functional.silu(y) if mode == 1 else pj[:, C:2 * C] * y).to(proj.dtype)
        state[page] = full[n:n + L - 1].to(state.dtype)
    return out


def short_conv(proj: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor], state: torch.Tensor,
               block_table: torch.Tensor, cu_q: Optional[torch.Tensor], q_per_seq: int, positions: torch.Tensor,
               slots: torch.Tensor, max_q_len: int = 1, mode: int = 0, x_off: int = 0) -> torch.Tensor:
    """proj [M, 3C] (mode 0) or [M, >= x_off + C] (mode 1) -> out [M, C]; ``state`` [pages, L-1, C] is updated in place.
    w fp32 [C, L]; column 0 of ``block_table`` names each sequence's state row."""
    if not proj.is_cuda:
        return short_conv_ref(proj, w, bias, state, block_table, cu_q, q_per_seq, positions, slots, mode, x_off)
    M = proj.shape[0]
    C, L = w.shape
    assert proj.dtype == torch.bfloat16 and state.dtype == torch.bfloat16 and proj.stride(1) == 1
    assert w.dtype == torch.float32 and w.is_contiguous() and state.is_contiguous() and slots.dtype == torch.int64
    out = torch.empty((M, C), dtype=proj.dtype, device=proj.device)
    B = block_table.shape[0]
    code = lib().eredu_short_conv(ptr(proj), proj.stride(0), ptr(w), ptr(bias), ptr(state), ptr(block_table),
                                  block_table.stride(0), ptr(cu_q), q_per_seq, ptr(positions), ptr(slots), ptr(out), C, L,
                                  B, max_q_len, mode, x_off, stream_ptr(proj.device))
    check(code, "eredu_short_conv")
    return out


native.register("eredu_conv_project", I, [P] * 19 + [I] * 20 + [P])


@dataclass
class ConvHeads:
    """Leading channels [q heads | k heads | v heads] of a projection: convolved, q and k rotated, q scaled per head, keys and
    values appended to the paged cache (and the means of the blocks of ``pool`` tokens they complete)."""
    taps: torch.Tensor                    # fp32 [taps, n_q dk + n_kv (dk + dv)]
    n_q: int
    n_kv: int
    dk: int
    dv: int
    inv_freq: torch.Tensor                # fp32 [rotated dims / 2]; neighbouring dims (2 i, 2 i + 1) form a pair
    k_cache: torch.Tensor
    v_cache: torch.Tensor
    q_scale: Optional[torch.Tensor] = None   # fp32 [n_q]
    pool: int = 0
    pooled: Optional[tuple] = None        # mean keys and values of the layer
    hist: int = 0                         # where the history starts in a sequence's state

    @property
    def channels(self) -> int:
        return self.taps.shape[1]


@dataclass
class ConvChannels:
    """``width`` channels of a projection from column ``start``: convolved, bias, SiLU."""
    taps: torch.Tensor                    # fp32 [taps, width]
    bias: Optional[torch.Tensor]          # fp32 [width]
    start: int
    hist: int = 0

    @property
    def width(self) -> int:
        return self.taps.shape[1]


def _conv_rows(u, taps, hist):
    """u [n, C] fp32, taps [L, C], hist [L - 1, C] -> (y [n, C], the new history)."""
    full = torch.cat((hist, u))
    return sum(taps[j] * full[j:j + u.shape[0]] for j in range(taps.shape[0])), full[full.shape[0] - hist.shape[0]:]


def conv_project_ref(proj, state, batch, page_to_slot, heads=None, channels=None):
    M = proj.shape[0]
    bounds = _sequences(batch)
    q = torch.zeros((M, heads.n_q, heads.dk), dtype=proj.dtype, device=proj.device) if heads is not None else None
    out = torch.zeros((M, channels.width), dtype=proj.dtype, device=proj.device) if channels is not None else None
    for b in range(len(bounds) - 1):
        r0, r1 = bounds[b], bounds[b + 1]
        if r1 <= r0 or int(batch.slots[r0]) < 0:
            continue
        st = state[int(page_to_slot[int(batch.block_table[b, 0])])].view(-1)
        for sec, start in ((heads, 0), (channels, channels.start if channels is not None else 0)):
            if sec is None:
                continue
            L, C = sec.taps.shape
            hist = st[sec.hist:sec.hist + (L - 1) * C].view(L - 1, C)
            y, new = _conv_rows(proj[r0:r1, start:start + C].float(), sec.taps.float(), hist.clone())
            hist.copy_(new)
            if sec is channels:
                y = y if sec.bias is None else y + sec.bias.float()
                out[r0:r1] = torch.nn.functional.silu(y).to(out.dtype)
                continue
            n, kw = sec.n_q * sec.dk, sec.n_kv * sec.dk
            rot = 2 * sec.inv_freq.shape[0]
            ang = batch.positions[r0:r1].float()[:, None] * sec.inv_freq.float()[None, :]
            cos, sin = ang.cos()[:, None, :], ang.sin()[:, None, :]

            def rotate(t):
                u, v = t[..., 0:rot:2], t[..., 1:rot:2]
                return torch.cat((torch.stack((u * cos - v * sin, v * cos + u * sin), -1).flatten(-2), t[..., rot:]), -1)

            qq = rotate(y[:, :n].view(-1, sec.n_q, sec.dk))
            if sec.q_scale is not None:
                qq = qq * sec.q_scale.float()[None, :, None]
            q[r0:r1] = qq.to(q.dtype)
            k, v = rotate(y[:, n:n + kw].view(-1, sec.n_kv, sec.dk)), y[:, n + kw:].view(-1, sec.n_kv, sec.dv)
            slots = batch.slots[r0:r1].long()
            sec.k_cache[slots // PAGE, :, slots % PAGE] = k.to(sec.k_cache.dtype)
            sec.v_cache[slots // PAGE, :, slots % PAGE] = v.to(sec.v_cache.dtype)
            if sec.pool:
                end = int(batch.seq_lens[b])
                for blk in range((end - (r1 - r0)) // sec.pool, end // sec.pool):
                    pool_block_ref(sec.k_cache, sec.v_cache, sec.pooled, batch.block_table[b], blk, sec.pool)
    return q, out


def conv_project(proj, state, batch, page_to_slot, heads: Optional[ConvHeads] = None, channels: Optional[ConvChannels] = None):
    """Causal depthwise convolutions ``y_t = sum_j taps[j] u_(t - L + 1 + j)`` over ranges of a projection's columns, one launch for
    both kinds of range: ``heads`` -> queries [M, n_q, dk], keys and values into their pages; ``channels`` -> silu(y + bias) [M, width].
    The last L - 1 inputs of a sequence live in ``state`` (fp32 [slots, ...]) from element ``hist`` on, [L - 1, channels]; zeros for a
    new sequence. Portions may have any length. Returns (queries or None, channels or None)."""
    if not proj.is_cuda:
        return conv_project_ref(proj, state, batch, page_to_slot, heads, channels)
    assert proj.stride(1) == 1 and state.is_contiguous() and state.dtype == torch.float32
    M, fp32 = proj.shape[0], proj.dtype == torch.float32
    q = out = None
    a, c = heads, channels
    if a is not None:
        assert a.k_cache.is_contiguous() and a.v_cache.is_contiguous() and a.k_cache.dtype == proj.dtype and a.taps.is_contiguous()
        q = torch.empty((M, a.n_q, a.dk), dtype=proj.dtype, device=proj.device)
    if c is not None:
        assert c.taps.is_contiguous()
        out = torch.empty((M, c.width), dtype=proj.dtype, device=proj.device)
    if M == 0:
        return q, out
    n = batch.block_table.shape[0]
    rows = batch.max_q_len if batch.is_prefill else batch.q_per_seq
    pk, pv = a.pooled if a is not None and a.pool else (None, None)
    code = lib().eredu_conv_project(
        ptr(proj), ptr(state), ptr(q), ptr(out), ptr(a.taps) if a else None, ptr(c.taps) if c else None, ptr(c.bias) if c else None,
        ptr(a.k_cache) if a else None, ptr(a.v_cache) if a else None, ptr(pk), ptr(pv), ptr(a.inv_freq) if a else None,
        ptr(a.q_scale) if a else None, ptr(batch.positions), ptr(batch.block_table), ptr(page_to_slot),
        ptr(batch.cu_q) if batch.is_prefill else None, ptr(batch.slots), ptr(batch.seq_lens), proj.stride(0), state[0].numel(),
        a.taps.shape[0] if a else 0, c.taps.shape[0] if c else 0, a.n_q if a else 0, a.n_kv if a else 0, a.dk if a else 0, a.dv if a else 0,
        2 * a.inv_freq.shape[0] if a else 0, a.pool if a else 0, pk.shape[2] if pk is not None else 0, a.hist if a else 0,
        c.width if c else 0, c.start if c else 0, c.hist if c else 0, n, batch.q_per_seq, rows, batch.block_table.stride(0),
        1 if fp32 else 0, stream_ptr(proj.device))
    check(code, "eredu_conv_project")
    return q, out


native.register("eredu_stream_conv", I, [P] * 8 + [I] * 8 + [P])


@dataclass
class StreamConv:
    """A causal convolution over the residual stream itself, in front of a sublayer. ``state`` [slots, >= (L - 1) W] starts with the last
    L - 1 inputs of a sequence, oldest first (None: one tap needs none)."""
    taps: torch.Tensor                    # fp32 [L, W], the last one multiplies the position itself
    state: Optional[torch.Tensor]
    batch: object                         # ForwardBatch
    page_to_slot: Optional[torch.Tensor]

    def checked(self, width: int):
        """(taps, state) as the kernels read them."""
        t, s = self.taps, self.state
        assert t.dtype == torch.float32 and t.is_contiguous() and t.shape[1] == width
        if t.shape[0] == 1:
            return t, None
        assert s.dtype == torch.float32 and s.is_contiguous() and s[0].numel() >= (t.shape[0] - 1) * width
        return t, s


def stream_conv_ref(x, conv, act_dtype):
    L, W = conv.taps.shape
    out = torch.zeros(x.shape, dtype=act_dtype, device=x.device)
    bounds = _sequences(conv.batch)
    for b in range(len(bounds) - 1):
        r0, r1 = bounds[b], bounds[b + 1]
        if r1 <= r0 or int(conv.batch.slots[r0]) < 0:
            continue
        hist = x.new_zeros(0, W)
        if L > 1:
            hist = conv.state[int(conv.page_to_slot[int(conv.batch.block_table[b, 0])])].view(-1)[:(L - 1) * W].view(L - 1, W)
        y, new = _conv_rows(x[r0:r1].float(), conv.taps.float(), hist.clone())
        hist.copy_(new)
        out[r0:r1] = (x[r0:r1] + y).to(act_dtype)
    return out


def stream_conv(x, conv: StreamConv, act_dtype):
    """``x_t + sum_j taps[j] x_(t - L + 1 + j)`` on every channel of the fp32 stream [M, W], in ``act_dtype``; zeros in front of a sequence's
    first token. The history in ``conv.state`` moves on. Portions may have any length."""
    if not x.is_cuda:
        return stream_conv_ref(x, conv, act_dtype)
    M, W = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous() and act_dtype in (torch.bfloat16, torch.float32)
    out = torch.empty((M, W), dtype=act_dtype, device=x.device)
    if M == 0:
        return out
    taps, state = conv.checked(W)
    b = conv.batch
    code = lib().eredu_stream_conv(
        ptr(x), ptr(out), ptr(taps), ptr(state), ptr(b.block_table), ptr(conv.page_to_slot) if state is not None else None,
        ptr(b.cu_q) if b.is_prefill else None, ptr(b.slots), b.block_table.shape[0], b.q_per_seq, b.max_q_len if b.is_prefill else b.q_per_seq,
        b.block_table.stride(0), W, taps.shape[0], state[0].numel() if state is not None else 0, 1 if act_dtype == torch.float32 else 0,
        stream_ptr(x.device))
    check(code, "eredu_stream_conv")
    return out
