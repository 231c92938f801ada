"""Mean keys and values of blocks of cached tokens, for attention that sees whole blocks behind its window.

Block b holds the positions b P .. b P + P - 1. Its means (over the rows as the cache holds them) live beside the page its last
position lies in: page ``(b P + P - 1) // 16`` of the sequence, row ``b - 16 page // P`` among the ``ceil(16 / P)`` rows of that page,
so they are given out and back with the page. A block's means are written when its last token is appended.
"""
from __future__ import annotations

import torch

from . import native
from .core import CLUSTER_SPLITS, _gather_kv, _tensor_core_dims
from .native import F, I, P, check, lib, ptr, status_word, stream_ptr

native.register("eredu_pool_blocks", I, [P] * 10 + [I] * 9 + [P])
native.register("eredu_attn_prefill_tc_pooled", I, [P] * 10 + [I] * 12 + [F, P, P])
native.register("eredu_attn_decode_pooled", I, [P] * 8 + [I] * 11 + [F, P])
native.register("eredu_attn_simt_pooled", I, [P] * 9 + [I] * 12 + [F, P])

PAGE = 16


def pooled_row(block: int, pool: int) -> tuple:
    """(page of the sequence, row in the page's means) of a block."""
    page = (block * pool + pool - 1) // PAGE
    return page, block - page * PAGE // pool


def pool_block_ref(k_cache, v_cache, pooled, table, block: int, pool: int) -> None:
    """Means of one block from the cached rows of the sequence with this row of the block table."""
    pos = torch.arange(block * pool, (block + 1) * pool, device=k_cache.device)
    page, row = pooled_row(block, pool)
    pages = table.long()[pos // PAGE]
    for cache, means in zip((k_cache, v_cache), pooled):
        means[int(table[page]), :, row] = cache[pages, :, pos % PAGE].float().mean(0).to(means.dtype)


def gather_pooled(pooled, table, blocks: int, pool: int) -> tuple:
    """The means of the first ``blocks`` blocks, (keys, values) [heads, blocks, width]."""
    rows = [pooled_row(b, pool) for b in range(blocks)]
    pages = table.long()[torch.tensor([p for p, _ in rows], dtype=torch.long, device=table.device)]
    at = torch.tensor([r for _, r in rows], dtype=torch.long, device=table.device)
    return tuple(m[pages, :, at].transpose(0, 1) for m in pooled)


def pool_rows(batch, pool: int) -> tuple:
    """(first row of every sequence in a dense array of all whole blocks [B] int32 on the device, rows of the array) of a batch of
    prompt portions; stated once per batch."""
    known = batch.pool_rows.get(pool)
    if known is None:
        counts = [(start + n) // pool for start, n in batch.host_portions()]
        first = [sum(counts[:i]) for i in range(len(counts))]
        t = torch.tensor(first, dtype=torch.int32)
        if batch.seq_lens.is_cuda:
            t = t.pin_memory().to(batch.seq_lens.device, non_blocking=True)
        known = batch.pool_rows[pool] = (t, sum(counts))
    return known


def pool_blocks(k_cache, v_cache, pooled, batch, pool: int, dense: bool = True):
    """Prompt portions: means of the blocks the new tokens complete, written beside their pages, and (``dense``) all whole blocks of
    every sequence as dense rows (keys [rows, heads, dk], values [rows, heads, dv], first row of every sequence)."""
    first, rows = pool_rows(batch, pool)
    n_kv, dk, dv = k_cache.shape[1], k_cache.shape[3], v_cache.shape[3]
    dk_rows = dv_rows = None
    if dense and rows:
        dk_rows = torch.empty((rows, n_kv, dk), dtype=k_cache.dtype, device=k_cache.device)
        dv_rows = torch.empty((rows, n_kv, dv), dtype=k_cache.dtype, device=k_cache.device)
    most = max((start + n) // pool for start, n in batch.host_portions())
    if most:
        code = lib().eredu_pool_blocks(
            ptr(k_cache), ptr(v_cache), ptr(pooled[0]), ptr(pooled[1]), ptr(dk_rows), ptr(dv_rows), ptr(batch.block_table), ptr(batch.seq_lens),
            ptr(batch.cu_q), ptr(first), batch.block_table.shape[0], batch.block_table.stride(0), most, n_kv, dk, dv, pool, pooled[0].shape[2],
            1 if k_cache.dtype == torch.float32 else 0, stream_ptr(k_cache.device))
        check(code, "eredu_pool_blocks")
    return dk_rows, dv_rows, first


def pool_cached_blocks(kv, layer: int, pool: int, pages, tokens: int) -> None:
    """Means of all whole blocks of the first ``tokens`` cached tokens of the sequence with these pages (whose keys and values were
    put into the cache by other means than a forward pass)."""
    k, v = kv.layer(layer)
    table = torch.as_tensor(list(pages), dtype=torch.int32, device=k.device)
    for b in range(tokens // pool):
        pool_block_ref(k, v, kv.pooled[layer], table, b, pool)


def blocks_seen(position: int, window: int, pool: int) -> int:
    """Whole blocks that lie before the window of a query at this position."""
    return max(0, (position - window + 1) // pool)


def pooled_attention_ref(q, k_cache, v_cache, pooled, block_table, seq_lens, q_lens, scale, window, pool):
    group = q.shape[1] // k_cache.shape[1]
    out = torch.empty((q.shape[0], q.shape[1], v_cache.shape[3]), dtype=q.dtype, device=q.device)
    start = 0
    for b, (kv_len, n) in enumerate(zip(seq_lens.tolist(), q_lens)):
        blocks = blocks_seen(kv_len - 1, window, pool)
        k, v = _gather_kv(k_cache, block_table[b], kv_len), _gather_kv(v_cache, block_table[b], kv_len)
        mk, mv = gather_pooled(pooled, block_table[b], blocks, pool)
        k = torch.cat((mk, k), 1).float().repeat_interleave(group, dim=0)
        v = torch.cat((mv, v), 1).float().repeat_interleave(group, dim=0)
        at = torch.arange(kv_len - n, kv_len, device=q.device)[:, None]
        key, blk = torch.arange(kv_len, device=q.device)[None], torch.arange(blocks, device=q.device)[None]
        seen = torch.cat((blk * pool + pool - 1 <= at - window, (key <= at) & (key > at - window)), 1)
        s = torch.einsum("hqd,hkd->hqk", q[start:start + n].float().transpose(0, 1), k) * scale
        p = torch.softmax(s.masked_fill(~seen[None], float("-inf")), -1)
        out[start:start + n] = torch.einsum("hqk,hkd->hqd", p, v).transpose(0, 1).to(q.dtype)
        start += n
    return out


def pooled_attention(q, k_cache, v_cache, pooled, batch, scale: float, window: int, pool: int):
    """Causal attention of ``q`` [M, n_q, dk] over the paged cache: a query at position i sees the ``window`` newest tokens up to its
    own and, under the same softmax, the mean key and value of every block of ``pool`` tokens whose last position is i - window or
    before. Prompt portions also write the means of the blocks they complete. Returns [M, n_q, dv]."""
    assert window > 0 and pool > 0
    if not q.is_cuda:
        q_lens = (batch.cu_q[1:] - batch.cu_q[:-1]).tolist() if batch.is_prefill else [batch.q_per_seq] * batch.block_table.shape[0]
        return pooled_attention_ref(q, k_cache, v_cache, pooled, batch.block_table, batch.seq_lens, q_lens, scale, window, pool)
    n_q, dk = q.shape[1], q.shape[2]
    n_kv, dv = k_cache.shape[1], v_cache.shape[3]
    assert q.is_contiguous() and k_cache.is_contiguous() and v_cache.is_contiguous() and q.dtype == k_cache.dtype
    assert all(t.is_contiguous() and t.dtype == k_cache.dtype for t in pooled)
    pk, pv = pooled
    B, most = batch.block_table.shape[0], batch.block_table.stride(0)
    out = torch.empty((q.shape[0], n_q, dv), dtype=q.dtype, device=q.device)
    tc = _tensor_core_dims(q, k_cache, v_cache)
    if batch.is_prefill:
        kr, vr, first = pool_blocks(k_cache, v_cache, pooled, batch, pool, dense=tc)
        if tc:
            code = lib().eredu_attn_prefill_tc_pooled(
                ptr(q), ptr(k_cache), ptr(v_cache), ptr(kr), ptr(vr), ptr(out), ptr(batch.block_table), ptr(batch.seq_lens), ptr(batch.cu_q),
                ptr(first), B, q.shape[0], batch.max_q_len, most, k_cache.shape[0], 0 if kr is None else kr.shape[0], n_q, n_kv, dk, dv,
                window, pool, scale, ptr(status_word(q.device)), stream_ptr(q.device))
            check(code, "eredu_attn_prefill_tc_pooled")
            return out
    if tc and n_q // n_kv <= 32 and not batch.is_prefill:
        splits = min(batch.layer_splits(n_kv, window + batch.max_kv_len // pool), CLUSTER_SPLITS)
        code = lib().eredu_attn_decode_pooled(
            ptr(q), ptr(k_cache), ptr(v_cache), ptr(pk), ptr(pv), ptr(out), ptr(batch.block_table), ptr(batch.seq_lens), B, batch.q_per_seq,
            most, n_q, n_kv, dk, dv, splits, window, pool, pk.shape[2], scale, stream_ptr(q.device))
        check(code, "eredu_attn_decode_pooled")
        return out
    rows = batch.max_q_len if batch.is_prefill else batch.q_per_seq
    code = lib().eredu_attn_simt_pooled(
        ptr(q), ptr(k_cache), ptr(v_cache), ptr(pk), ptr(pv), ptr(out), ptr(batch.block_table), ptr(batch.seq_lens),
        ptr(batch.cu_q) if batch.is_prefill else None, B, batch.q_per_seq, rows, most, n_q, n_kv, dk, dv, window, pool, pk.shape[2],
        1 if q.dtype == torch.float32 else 0, scale, stream_ptr(q.device))
    check(code, "eredu_attn_simt_pooled")
    return out
