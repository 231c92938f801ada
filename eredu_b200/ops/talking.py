"""Attention whose heads exchange their scores before the softmax (Shazeer, Lan, Cheng, Ding, Hou: "Talking-Heads Attention"; the
mixing in front of the softmax only)."""
from __future__ import annotations

import torch

from . import native
from .core import CLUSTER_SPLITS, PAGE, _gather_kv, _sm_count, _tensor_core_dims
from .native import F, I, P, check, lib, ptr, status_word, stream_ptr

native.register("eredu_talking_attention", I, [P] * 9 + [I] * 12 + [F, F, P, P])
native.register("eredu_talking_attention_simt", I, [P] * 9 + [I] * 11 + [F, F, P])
native.register("eredu_talking_fits", I, [I] * 5)


def visible_keys(qpos, kpos, window: int, keep: int):
    """Causal; with a ``window`` the newest ``window`` positions up to the query's own and the first ``keep`` of the sequence."""
    seen = kpos <= qpos
    return seen & ((qpos - kpos < window) | (kpos < keep)) if window > 0 else seen


def talking_attention_ref(q, k_cache, v_cache, block_table, seq_lens, q_lens, talk, scale, softcap, sinks=None, window=0, keep=0):
    group = q.shape[1] // k_cache.shape[1]
    out = torch.empty((q.shape[0], q.shape[1], v_cache.shape[3]), dtype=q.dtype, device=q.device)
    start = 0
    for b, (kv_len, n) in enumerate(zip(seq_lens.tolist(), q_lens)):
        k, v = (_gather_kv(c, block_table[b], kv_len).float().repeat_interleave(group, dim=0) for c in (k_cache, v_cache))
        s = torch.einsum("hqd,hkd->hqk", q[start:start + n].float().transpose(0, 1), k) * scale
        if softcap > 0:
            s = softcap * torch.tanh(s / softcap)
        s = torch.einsum("hg,gqk->hqk", talk.float(), s)
        seen = visible_keys(torch.arange(kv_len - n, kv_len, device=q.device)[:, None], torch.arange(kv_len, device=q.device)[None], window, keep)
        s = s.masked_fill(~seen[None], float("-inf"))
        if sinks is not None:
            s = torch.cat((s, sinks.float()[:, None, None].expand(-1, n, 1)), -1)
        p = torch.softmax(s, -1)[..., :kv_len]
        out[start:start + n] = torch.einsum("hqk,hkd->hqd", p, v).transpose(0, 1).to(q.dtype)
        start += n
    return out


def talking_attention(q, k_cache, v_cache, batch, talk, scale: float, softcap: float = 0.0, sinks=None, window: int = 0, keep: int = 0):
    """Causal attention of ``q`` [M, H, dk] over the paged cache. The score of head h is ``sum_g talk[h, g] * cap(scale * q_g . k_g)`` with
    ``cap(s) = softcap * tanh(s / softcap)`` (no cap: 0); the softmax over the visible keys has one more term exp(sinks[h]) in its
    denominator. ``window``, ``keep``: :func:`visible_keys`. ``talk`` [H, H] in q's dtype, ``sinks`` fp32 [H]. Returns [M, H, dv]."""
    if not q.is_cuda:
        q_lens = (batch.cu_q[1:] - batch.cu_q[:-1]).tolist() if batch.is_prefill else [batch.q_per_seq] * batch.block_table.shape[0]
        return talking_attention_ref(q, k_cache, v_cache, batch.block_table, batch.seq_lens, q_lens, talk, scale, softcap, sinks, window, keep)
    H, G, dk, dv = q.shape[1], k_cache.shape[1], q.shape[2], v_cache.shape[3]
    assert q.is_contiguous() and k_cache.is_contiguous() and v_cache.is_contiguous() and q.dtype == k_cache.dtype == v_cache.dtype
    assert talk.dtype == q.dtype and talk.is_contiguous() and talk.shape == (H, H) and (sinks is None or sinks.dtype == torch.float32)
    out = torch.empty((q.shape[0], H, dv), dtype=q.dtype, device=q.device)
    if q.shape[0] == 0:
        return out
    B, rows = batch.block_table.shape[0], batch.max_q_len if batch.is_prefill else batch.q_per_seq
    args = (ptr(q), ptr(k_cache), ptr(v_cache), ptr(out), ptr(batch.block_table), ptr(batch.seq_lens), ptr(batch.cu_q) if batch.is_prefill else None,
            ptr(talk), ptr(sinks), B, batch.q_per_seq, rows, batch.block_table.stride(0), H, G, dk, dv, window, keep)
    if _tensor_core_dims(q, k_cache, v_cache) and lib().eredu_talking_fits(H, G, dk, dv, rows):
        splits = 1 if batch.is_prefill else decode_splits(B, batch.max_kv_len, window, keep, _sm_count(q.device))
        check(lib().eredu_talking_attention(*args, splits, k_cache.shape[0], scale, softcap, ptr(status_word(q.device)), stream_ptr(q.device)), "eredu_talking_attention")
        return out
    check(lib().eredu_talking_attention_simt(*args, 1 if q.dtype == torch.float32 else 0, scale, softcap, stream_ptr(q.device)),
          "eredu_talking_attention_simt")
    return out


def decode_splits(batch: int, max_kv_len: int, window: int, keep: int, sm_count: int) -> int:
    """CTAs that share the keys of one sequence in a decode step: the machine filled once, at least four pages each, at most as many as
    one cluster combines."""
    seen = min(max_kv_len, window + keep + PAGE) if window > 0 else max_kv_len
    return max(1, min(sm_count // max(1, batch), -(-seen // PAGE) // 4, CLUSTER_SPLITS))
