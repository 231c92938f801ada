"""Recurrent scans of hybrid (linear-attention) layers.

``gated_delta_scan``: the gated delta rule (eredu/src/backend/mlx/nn/gated_delta.rs:135-183 step, :295-360 scan)::

    S <- S * exp(g_t);  m = S^T k_t;  S <- S + k_t (beta_t (v_t - m))^T;  o_t = S^T q_t

with the state ``S [B, H, Dk, Dv]`` in fp32. ``log_decay`` is ``[B, T, H]`` (one decay per head) or ``[B, T, H, Dk]`` (one
per key channel). Feeding a sequence in chunks with the returned state gives the same outputs as one scan.
"""
from __future__ import annotations

from typing import Optional

import torch

from . import native
from .core import _sm_count
from .native import F, I, P, check, lib, ptr, stream_ptr

native.register("eredu_gated_delta_scan", I, [P, P, P, P, P, P, P, I, I, I, I, I, I, P])
native.register("eredu_mamba2_scan", I, [P, P, P, P, P, P, P, P, I, I, I, I, I, I, P])
native.register("eredu_mingru_scan", I, [P] * 8 + [I] * 7 + [P])
native.register("eredu_mingru_scratch_elems", native.L, [I] * 4)
native.register("eredu_gla_scan", I, [P] * 7 + [I] + [P] * 4 + [I] * 10 + [F, F, P])
native.register("eredu_gla_scratch_elems", native.L, [I] * 8)


# From this many tokens per call the chunk-parallel Mamba-2 form takes over from the token-by-token kernel (measured on a
# B200, 64 heads x 64, state 128: 1.15x at 2048 tokens, 2.5x at 8192). The gated-delta form is exact but, as a chain of
# small library calls (triangular solve, three GEMMs per chunk), 2.5-5x slower than the kernel at those lengths: it is
# not dispatched to.
CHUNKED_SCAN_MIN_TOKENS = 2048


def gated_delta_scan_ref(q, k, v, log_decay, beta, state: Optional[torch.Tensor] = None):
    """PyTorch reference; returns (state fp32 [B, H, Dk, Dv], out [B, T, H, Dv] in q's dtype)."""
    if q.dim() != 4 or k.dim() != 4 or v.dim() != 4:
        raise ValueError("gated-delta query, key and value tensors must be rank 4")
    if q.shape[:3] != k.shape[:3] or q.shape[:3] != v.shape[:3] or q.shape[3] != k.shape[3]:
        raise ValueError("gated-delta query, key and value batch / sequence / head dimensions must match")
    B, T, H, Dk = q.shape
    Dv = v.shape[-1]
    if log_decay.dim() not in (3, 4) or tuple(log_decay.shape[:3]) != (B, T, H) or (log_decay.dim() == 4 and log_decay.shape[3] != Dk):
        raise ValueError(f"gated-delta log decay shape {tuple(log_decay.shape)} is incompatible with query shape {tuple(q.shape)}")
    if tuple(beta.shape) != (B, T, H):
        raise ValueError(f"gated-delta beta shape {tuple(beta.shape)} must equal {(B, T, H)}")
    S = torch.zeros((B, H, Dk, Dv), dtype=torch.float32, device=q.device) if state is None else state.float().clone()
    if tuple(S.shape) != (B, H, Dk, Dv):
        raise ValueError(f"gated-delta state shape {tuple(S.shape)} must equal {(B, H, Dk, Dv)}")
    outs = []
    qf, kf, vf, bf = q.float(), k.float(), v.float(), beta.float()
    decay = torch.exp(log_decay.float())
    for t in range(T):
        d = decay[:, t]
        d = d[:, :, None, None] if d.dim() == 2 else d[:, :, :, None]
        S = S * d
        kt = kf[:, t][..., None]                                  # [B, H, Dk, 1]
        mem = (S * kt).sum(-2)                                    # [B, H, Dv]
        delta = (vf[:, t] - mem) * bf[:, t][..., None]
        S = S + kt * delta[:, :, None, :]
        outs.append((S * qf[:, t][..., None]).sum(-2))
    return S, torch.stack(outs, 1).to(q.dtype)


def gated_delta_scan_chunked(q, k, v, log_decay, beta, state: Optional[torch.Tensor] = None, chunk: int = 64, gemm_dtype=None):
    """The gated delta rule with one decay per head and step in its chunk-parallel form. With ``gamma_t`` the decay
    accumulated since the start of the chunk, the state inside a chunk is ``S_t = gamma_t S_0 + sum_{s <= t}
    (gamma_t / gamma_s) k_s u_s^T`` for pseudo-values ``u`` that solve a unit lower-triangular system
    ``(I + diag(beta) A) U = diag(beta) (V - diag(gamma) K S_0)``, ``A[t, s] = (gamma_t / gamma_s) k_t . k_s`` for
    ``s < t``. The inverse and its products with ``V`` and ``K`` are computed for all chunks at once; what stays
    sequential is one step per chunk with three GEMMs (``U``, the outputs, the state). Same arguments and results as
    :func:`gated_delta_scan_ref` (``log_decay`` of shape [B, T, H] only)."""
    if log_decay.dim() != 3:
        raise ValueError("the chunk-parallel form takes one decay per head and step")
    B_, T, H, Dk = q.shape
    Dv = v.shape[-1]
    dev = q.device
    gd = gemm_dtype or (torch.bfloat16 if q.is_cuda else torch.float32)
    S = torch.zeros((B_, H, Dk, Dv), dtype=torch.float32, device=dev) if state is None else state.float().clone()
    Qn = int(chunk)
    nc = (T + Qn - 1) // Qn
    pad = nc * Qn - T

    def prep(t, width=None):                   # [B, T, H, (W)] -> [B, H, nc, Q, (W)] fp32, zero padded
        t = t.float()
        if pad:
            t = torch.cat((t, t.new_zeros((B_, pad) + tuple(t.shape[2:]))), 1)
        t = t.view(B_, nc, Qn, *t.shape[2:])
        return t.permute(0, 3, 1, 2, 4) if t.dim() == 5 else t.permute(0, 3, 1, 2)

    qf, kf, vf = prep(q), prep(k), prep(v)
    bf, a = prep(beta), prep(log_decay)                                 # padded steps: beta 0, decay 1, key 0
    L = torch.cumsum(a, -1)                                             # log gamma_t, inclusive
    gamma = torch.exp(L)
    diff = L[..., :, None] - L[..., None, :]
    tri = torch.ones((Qn, Qn), dtype=torch.bool, device=dev).tril()
    ratio = torch.where(tri, torch.exp(diff.masked_fill(~tri, 0.0)), torch.zeros((), device=dev))          # gamma_t / gamma_s, s <= t
    kk = torch.matmul(kf.to(gd), kf.to(gd).transpose(-1, -2)).float()   # [B, H, nc, Q, Q]
    strict = torch.ones((Qn, Qn), dtype=torch.bool, device=dev).tril(-1)
    A = torch.where(strict, ratio * kk, torch.zeros((), device=dev)) * bf[..., None]
    eye = torch.eye(Qn, device=dev)
    Tm = torch.linalg.solve_triangular(eye + A, eye.expand_as(A).contiguous(), upper=False, unitriangular=True)
    Wv = torch.matmul(Tm, vf * bf[..., None])                           # [B, H, nc, Q, Dv]
    Wk = torch.matmul(Tm, kf * (bf * gamma)[..., None])                 # [B, H, nc, Q, Dk]
    qk = torch.matmul(qf.to(gd), kf.to(gd).transpose(-1, -2)).float() * ratio                               # s <= t
    to_end = torch.exp(L[..., -1:] - L)                                 # gamma_Q / gamma_s
    kend = kf * to_end[..., None]
    outs = []
    for c in range(nc):
        U = Wv[:, :, c] - torch.matmul(Wk[:, :, c].to(gd), S.to(gd)).float()                               # [B, H, Q, Dv]
        o = torch.matmul(qf[:, :, c].to(gd), S.to(gd)).float() * gamma[:, :, c, :, None] + torch.matmul(qk[:, :, c].to(gd), U.to(gd)).float()
        S = S * gamma[:, :, c, -1, None, None] + torch.matmul(kend[:, :, c].to(gd).transpose(-1, -2), U.to(gd)).float()
        outs.append(o)
    out = torch.stack(outs, 2).permute(0, 2, 3, 1, 4).reshape(B_, nc * Qn, H, Dv)[:, :T]
    return S, out.to(q.dtype)


def gated_delta_scan(q, k, v, log_decay, beta, state: Optional[torch.Tensor] = None):
    """CUDA: one kernel for the whole chunk (bf16 q / k / v, Dk of 64 or 128); otherwise the reference."""
    if not q.is_cuda or q.dtype != torch.bfloat16 or q.shape[-1] not in (64, 128):
        return gated_delta_scan_ref(q, k, v, log_decay, beta, state)
    B, T, H, Dk = q.shape
    Dv = v.shape[-1]
    if tuple(beta.shape) != (B, T, H) or tuple(log_decay.shape[:3]) != (B, T, H):
        raise ValueError("gated-delta beta / log decay shapes do not match the query")
    S = torch.zeros((B, H, Dk, Dv), dtype=torch.float32, device=q.device) if state is None else state.float().contiguous().clone()
    out = torch.empty((B, T, H, Dv), dtype=q.dtype, device=q.device)
    # every operand is bound to a name until the launch is queued: a temporary made by ``.contiguous()`` / ``.float()``
    # would go back to the caching allocator at once and the next temporary could land on the same bytes
    g = log_decay.float().contiguous()
    qc, kc, vc, bc = q.contiguous(), k.to(q.dtype).contiguous(), v.to(q.dtype).contiguous(), beta.float().contiguous()
    code = lib().eredu_gated_delta_scan(ptr(qc), ptr(kc), ptr(vc), ptr(g), ptr(bc), ptr(S), ptr(out), B, T, H, Dk, Dv,
                                        1 if g.dim() == 4 else 0, stream_ptr(q.device))
    check(code, "eredu_gated_delta_scan")
    return S, out


def mamba2_scan_ref(x, B, C, dt, A, D, state: Optional[torch.Tensor] = None):
    """Mamba-2 selective state-space recurrence, token by token (eredu/src/backend/mlx/architectures/nemotron_h/
    model.rs:1929-1962): ``S <- S * exp(dt A) + x (dt B)^T;  y = S C + D x`` per head.

    x [Bt, T, H, P]; B, C [Bt, T, G, N] with G dividing H (one B / C per group of heads; G = H when already expanded);
    dt [Bt, T, H] (after softplus and floor); A [H] (negative); D [H]; state fp32 [Bt, H, P, N]. Returns (state,
    y [Bt, T, H, P] in x's dtype)."""
    Bt, T, H, P = x.shape
    N = B.shape[-1]
    if B.shape[2] != H:
        if H % B.shape[2]:
            raise ValueError("Mamba-2 group count must divide the head count")
        B, C = B.repeat_interleave(H // B.shape[2], 2), C.repeat_interleave(H // C.shape[2], 2)
    S = torch.zeros((Bt, H, P, N), dtype=torch.float32, device=x.device) if state is None else state.float().clone()
    xf, Bf, Cf, dtf = x.float(), B.float(), C.float(), dt.float()
    Af, Df = A.float().view(1, H, 1, 1), D.float().view(1, H, 1)
    ys = []
    for t in range(T):
        d = dtf[:, t]                                                     # [Bt, H]
        dA = torch.exp(d[:, :, None, None] * Af)
        dBx = xf[:, t][..., None] * (d[:, :, None] * Bf[:, t])[:, :, None, :]
        S = S * dA + dBx
        ys.append((S * Cf[:, t][:, :, None, :]).sum(-1) + xf[:, t] * Df)
    return S, torch.stack(ys, 1).to(x.dtype)


def mamba2_scan_chunked(x, B, C, dt, A, D, state: Optional[torch.Tensor] = None, chunk: int = 64, gemm_dtype=None):
    """The same recurrence in its chunk-parallel (state-space duality) form: the sequence is cut into chunks of ``chunk``
    tokens; inside a chunk the outputs are a masked, decay-weighted ``(C B^T) x`` product, every chunk contributes one
    state update ``sum_s decay(s -> end) x_s B_s^T``, the states are carried from chunk to chunk (the only sequential
    part: T / chunk steps on [P, N] matrices) and enter the outputs as ``decay(start -> t) C_t S``. All four products
    are batched GEMMs, so a long prefill runs on the tensor cores instead of token by token. Same arguments and results
    as :func:`mamba2_scan_ref`; ``gemm_dtype`` (default: fp32 on the CPU, bf16 on CUDA) is the operand type of the
    GEMMs, decays and accumulation stay fp32."""
    Bt, T, H, P = x.shape
    G, N = B.shape[2], B.shape[3]
    if H % G:
        raise ValueError("Mamba-2 group count must divide the head count")
    dev = x.device
    gd = gemm_dtype or (torch.bfloat16 if x.is_cuda else torch.float32)
    S = torch.zeros((Bt, H, P, N), dtype=torch.float32, device=dev) if state is None else state.float().clone()
    Q = int(chunk)
    nc = (T + Q - 1) // Q
    pad = nc * Q - T
    xf, dtf = x.float(), dt.float()
    if pad:                                   # padded steps have dt = 0: no decay, no input, outputs dropped
        xf = torch.cat((xf, xf.new_zeros(Bt, pad, H, P)), 1)
        dtf = torch.cat((dtf, dtf.new_zeros(Bt, pad, H)), 1)
        B = torch.cat((B, B.new_zeros(Bt, pad, G, N)), 1)
        C = torch.cat((C, C.new_zeros(Bt, pad, G, N)), 1)
    rep = H // G
    a = dtf * A.float().view(1, 1, H)                                   # log decay per step, <= 0
    a = a.view(Bt, nc, Q, H).permute(0, 3, 1, 2)                        # [Bt, H, nc, Q]
    L = torch.cumsum(a, -1)                                             # inclusive prefix inside the chunk
    xs = (xf * dtf[..., None]).view(Bt, nc, Q, H, P).permute(0, 3, 1, 2, 4)            # x * dt: [Bt, H, nc, Q, P]
    Bc = B.float().view(Bt, nc, Q, G, N).permute(0, 3, 1, 2, 4)         # [Bt, G, nc, Q, N]
    Cc = C.float().view(Bt, nc, Q, G, N).permute(0, 3, 1, 2, 4)
    # inside a chunk: y[t] = sum_{s <= t} exp(L_t - L_s) (C_t . B_s) xs[s]
    cb = torch.matmul(Cc.to(gd), Bc.to(gd).transpose(-1, -2)).float()   # [Bt, G, nc, Q, Q]
    cb = cb.repeat_interleave(rep, 1) if rep > 1 else cb                # [Bt, H, nc, Q, Q]
    diff = L[..., :, None] - L[..., None, :]                            # L_t - L_s
    tri = torch.ones((Q, Q), dtype=torch.bool, device=dev).tril()
    w = torch.where(tri, torch.exp(diff.masked_fill(~tri, 0.0)), torch.zeros((), device=dev)) * cb
    y = torch.matmul(w.to(gd), xs.to(gd)).float()                       # [Bt, H, nc, Q, P]
    # what every chunk adds to the state: sum_s exp(L_end - L_s) xs[s] B_s^T
    to_end = torch.exp(L[..., -1:] - L)                                 # [Bt, H, nc, Q]
    Bh = Bc.repeat_interleave(rep, 1) if rep > 1 else Bc                # [Bt, H, nc, Q, N]
    Ch = Cc.repeat_interleave(rep, 1) if rep > 1 else Cc
    upd = torch.matmul((xs * to_end[..., None]).to(gd).transpose(-1, -2), Bh.to(gd)).float()      # [Bt, H, nc, P, N]
    total = torch.exp(L[..., -1])                                       # decay over a whole chunk: [Bt, H, nc]
    # the sequential part: the state that enters every chunk
    entering = []
    for c in range(nc):
        entering.append(S)
        S = S * total[:, :, c, None, None] + upd[:, :, c]
    Sin = torch.stack(entering, 2)                                      # [Bt, H, nc, P, N]
    # contribution of the entering state: exp(L_t) C_t . S
    y = y + torch.matmul(Ch.to(gd), Sin.to(gd).transpose(-1, -2)).float() * torch.exp(L)[..., None]
    y = y.permute(0, 2, 3, 1, 4).reshape(Bt, nc * Q, H, P)[:, :T]
    y = y + xf[:, :T] * D.float().view(1, 1, H, 1)
    return S, y.to(x.dtype)


def mamba2_scan(x, B, C, dt, A, D, state: Optional[torch.Tensor] = None):
    """CUDA: one kernel for the whole chunk (bf16 x / B / C, state size 64, 128 or 256) for decode-sized calls, the
    chunk-parallel GEMM form for long prefills; otherwise the reference."""
    if x.is_cuda and x.shape[1] >= CHUNKED_SCAN_MIN_TOKENS:
        return mamba2_scan_chunked(x, B, C, dt, A, D, state)
    if not x.is_cuda or x.dtype != torch.bfloat16 or B.shape[-1] not in (64, 128, 256):
        return mamba2_scan_ref(x, B, C, dt, A, D, state)
    Bt, T, H, P_ = x.shape
    G, N = B.shape[2], B.shape[3]
    if tuple(C.shape) != tuple(B.shape) or tuple(B.shape[:2]) != (Bt, T) or H % G or tuple(dt.shape) != (Bt, T, H):
        raise ValueError("Mamba-2 B / C / dt shapes do not match x")
    S = torch.zeros((Bt, H, P_, N), dtype=torch.float32, device=x.device) if state is None else state.float().contiguous().clone()
    if tuple(S.shape) != (Bt, H, P_, N):
        raise ValueError(f"Mamba-2 state shape {tuple(S.shape)} must equal {(Bt, H, P_, N)}")
    out = torch.empty((Bt, T, H, P_), dtype=x.dtype, device=x.device)
    # operands stay bound to names until the launch is queued (see gated_delta_scan)
    xc, Bc, Cc = x.contiguous(), B.to(torch.bfloat16).contiguous(), C.to(torch.bfloat16).contiguous()
    dtc, Ac, Dc = dt.float().contiguous(), A.float().contiguous(), D.float().contiguous()
    code = lib().eredu_mamba2_scan(ptr(xc), ptr(Bc), ptr(Cc), ptr(dtc), ptr(Ac), ptr(Dc), ptr(S), ptr(out), Bt, T, H, G,
                                   P_, N, stream_ptr(x.device))
    check(code, "eredu_mamba2_scan")
    return S, out


# ---------------------------------------------------------------------------------------------- ragged recurrences
# The operators below take the rows of a whole batch - portions of prompts of any length beside single decoded tokens -
# and find each sequence's fp32 state on the device: state[page_to_slot[first page of the sequence]]. ``batch`` gives the
# rows of every sequence (``cu_q`` or ``q_per_seq`` each), the block table and the cache slots; a sequence whose first row has
# no cache slot (an idle row of a captured decode batch) leaves its state alone.
def _sequences(batch):
    B = batch.block_table.shape[0]
    return batch.cu_q.tolist() if batch.is_prefill else [i * batch.q_per_seq for i in range(B + 1)]


def mingru_scan_ref(proj, state, width, batch, page_to_slot):
    out = torch.zeros((proj.shape[0], width), dtype=proj.dtype, device=proj.device)
    z, u, g = (proj[:, i * width:(i + 1) * width].float() for i in range(3))
    z, cand = torch.sigmoid(z), torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    bounds = _sequences(batch)
    for b in range(len(bounds) - 1):
        r0, r1 = bounds[b], bounds[b + 1]
        if r1 <= r0 or int(batch.slots[r0]) < 0:
            continue
        slot = int(page_to_slot[int(batch.block_table[b, 0])])
        S = state[slot].clone()
        for t in range(r0, r1):
            S = (1 - z[t]) * S + z[t] * cand[t]
            out[t] = (S * torch.nn.functional.silu(g[t])).to(out.dtype)
        state[slot] = S
    return out


def mingru_scan(proj, state, width, batch, page_to_slot):
    """minGRU: ``proj`` [M, 3 width] = [z | u | gate]; ``S <- (1 - sigmoid(z)) S + sigmoid(z) c(u)`` with ``c(u) = u + 1/2``
    for u >= 0 and ``sigmoid(u)`` below, output ``S * silu(gate)`` [M, width]. ``state`` fp32 [slots, width], in place."""
    if not proj.is_cuda:
        return mingru_scan_ref(proj, state, width, batch, page_to_slot)
    assert proj.stride(1) == 1 and state.is_contiguous() and state.dtype == torch.float32
    out = torch.empty((proj.shape[0], width), dtype=proj.dtype, device=proj.device)
    if proj.shape[0] == 0:
        return out
    batch_size = batch.block_table.shape[0]
    rows = batch.max_q_len if batch.is_prefill else batch.q_per_seq
    elems = int(lib().eredu_mingru_scratch_elems(width, proj.shape[0], batch_size, rows))
    scratch = torch.empty(elems, dtype=torch.float32, device=proj.device) if elems else None
    code = lib().eredu_mingru_scan(ptr(proj), ptr(state), ptr(out), ptr(scratch), ptr(batch.block_table), ptr(page_to_slot),
                                   ptr(batch.cu_q) if batch.is_prefill else None, ptr(batch.slots), width, proj.stride(0),
                                   batch_size, batch.q_per_seq, rows, batch.block_table.stride(0),
                                   1 if proj.dtype == torch.float32 else 0, stream_ptr(proj.device))
    check(code, "eredu_mingru_scan")
    return out


def gla_scan_ref(q, k, v, log_decay, state):
    """q, k, log_decay [T, H, D], v [T, H, V], state [H, D, V] (all fp32): ``S <- diag(exp(log_decay)) S + k v^T``,
    ``o = S^T q``. Returns (o [T, H, V], state)."""
    S, out = state.clone(), []
    decay = torch.exp(log_decay)
    for t in range(q.shape[0]):
        S = S * decay[t][:, :, None] + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def gla_attention_ref(proj, a2, a2_b, norm_w, state, heads, dk, dv, tau, eps, batch, page_to_slot):
    M, qk, vw = proj.shape[0], heads * dk, heads * dv
    x = proj.float()
    q, k = x[:, :qk].view(M, heads, dk) * dk ** -0.5, x[:, qk:2 * qk].view(M, heads, dk)
    v, g = x[:, 2 * qk:2 * qk + vw].view(M, heads, dv), x[:, 2 * qk + vw:2 * qk + 2 * vw]
    z = x[:, 2 * qk + 2 * vw:] @ a2.t() + a2_b
    logd = (torch.nn.functional.logsigmoid(z) / tau).view(M, heads, dk)
    out = torch.zeros((M, vw), dtype=proj.dtype, device=proj.device)
    bounds = _sequences(batch)
    for b in range(len(bounds) - 1):
        r0, r1 = bounds[b], bounds[b + 1]
        if r1 <= r0 or int(batch.slots[r0]) < 0:
            continue
        slot = int(page_to_slot[int(batch.block_table[b, 0])])
        o, state[slot] = gla_scan_ref(q[r0:r1], k[r0:r1], v[r0:r1], logd[r0:r1], state[slot])
        o = o * torch.rsqrt(o.square().mean(-1, keepdim=True) + eps) * norm_w
        out[r0:r1] = (o.reshape(r1 - r0, vw) * torch.nn.functional.silu(g[r0:r1])).to(out.dtype)
    return out


def gla_attention(proj, a2, a2_b, norm_w, state, heads, dk, dv, tau, eps, batch, page_to_slot):
    """Gated linear attention over ``proj`` [M, 2 H dk + 2 H dv + r] = [q | k | v | gate | low-rank decay input]:
    per head ``S <- diag(alpha) S + k v^T``, ``o = S^T q / sqrt(dk)`` with ``alpha = sigmoid(a2 low + a2_b)^(1 / tau)`` per key
    channel; each head's o is RMS-normed (weight ``norm_w`` [dv]) and multiplied by ``silu(gate)``. ``a2`` fp32 [H dk, r];
    ``state`` fp32 [slots, H, dk, dv], in place. Returns [M, H dv]."""
    if not proj.is_cuda:
        return gla_attention_ref(proj, a2, a2_b, norm_w, state, heads, dk, dv, tau, eps, batch, page_to_slot)
    M = proj.shape[0]
    assert proj.stride(1) == 1 and state.is_contiguous() and state.dtype == torch.float32 and a2.is_contiguous()
    out = torch.empty((M, heads * dv), dtype=proj.dtype, device=proj.device)
    if M == 0:
        return out
    batch_size = batch.block_table.shape[0]
    rows = batch.max_q_len if batch.is_prefill else batch.q_per_seq
    scratch = None
    if proj.dtype == torch.bfloat16 and proj.data_ptr() % 16 == 0:
        elems = int(lib().eredu_gla_scratch_elems(heads, dk, dv, a2.shape[1], proj.stride(0), M, batch_size, rows))
        if elems:
            scratch = torch.empty(elems, dtype=torch.float32, device=proj.device)
    code = lib().eredu_gla_scan(ptr(proj), ptr(a2), ptr(a2_b), ptr(norm_w), ptr(state), ptr(out), ptr(scratch), M,
                                ptr(batch.block_table), ptr(page_to_slot), ptr(batch.cu_q) if batch.is_prefill else None,
                                ptr(batch.slots), heads, dk, dv, a2.shape[1], proj.stride(0), batch_size, batch.q_per_seq, rows,
                                batch.block_table.stride(0), 1 if proj.dtype == torch.float32 else 0, tau, eps,
                                stream_ptr(proj.device))
    check(code, "eredu_gla_scan")
    return out


native.register("eredu_mlstm", I, [P] * 10 + [I] * 13 + [F, F, P])
native.register("eredu_mlstm_scratch_bytes", native.L, [I] * 7)


def mlstm_state_views(state, heads, dk, dv):
    """One sequence's state [>= H (dk dv + dk + 1)] as (memory [H, dk, dv], normaliser [H, dk], running maximum [H])."""
    a, b = heads * dk * dv, heads * dk
    return state[:a].view(heads, dk, dv), state[a:a + b].view(heads, dk), state[a + b:a + b + heads]


def mlstm_scan_ref(q, k, v, i, f, state):
    """q, k [T, H, dk], v [T, H, dv], log gates i, f [T, H] (fp32); state (S, n, m). Returns (o [T, H, dv], state)."""
    S, n, m = (t.clone() for t in state)
    out = []
    for t in range(q.shape[0]):
        new = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        kt = k[t] * take[:, None]
        S = S * keep[:, None, None] + kt[:, :, None] * v[t][:, None, :]
        n = n * keep[:, None] + kt
        m = new
        size = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + MLSTM_EPS
        out.append(torch.einsum("hdv,hd->hv", S, q[t]) / size[:, None])
    return torch.stack(out), (S, n, m)


MLSTM_EPS = 1e-6        # added to the normaliser


def mlstm_ref(proj, gates, norm_w, state, heads, dk, dv, cap, eps, batch, page_to_slot):
    M, qk, vw = proj.shape[0], heads * dk, heads * dv
    x = proj.float()
    q, k = x[:, :qk].view(M, heads, dk) * dk ** -0.5, x[:, qk:2 * qk].view(M, heads, dk)
    v, g = x[:, 2 * qk:2 * qk + vw].view(M, heads, dv), x[:, 2 * qk + vw:2 * qk + 2 * vw]
    z = cap * torch.tanh(gates.float() / cap)
    i, f = z[:, :heads], torch.nn.functional.logsigmoid(z[:, heads:2 * heads])
    out = torch.zeros((M, vw), dtype=proj.dtype, device=proj.device)
    bounds = _sequences(batch)
    for b in range(len(bounds) - 1):
        r0, r1 = bounds[b], bounds[b + 1]
        if r1 <= r0 or int(batch.slots[r0]) < 0:
            continue
        views = mlstm_state_views(state[int(page_to_slot[int(batch.block_table[b, 0])])], heads, dk, dv)
        o, new = mlstm_scan_ref(q[r0:r1], k[r0:r1], v[r0:r1], i[r0:r1], f[r0:r1], views)
        for old, t in zip(views, new):
            old.copy_(t)
        o = (o * torch.rsqrt(o.square().mean(-1, keepdim=True) + eps)).reshape(r1 - r0, vw) * norm_w
        out[r0:r1] = (o * torch.sigmoid(g[r0:r1])).to(out.dtype)
    return out


def mlstm(proj, gates, norm_w, state, heads, dk, dv, cap, eps, batch, page_to_slot):
    """Matrix memory with exponential gates (mLSTM) over ``proj`` [M, >= 2 H dk + 2 H dv] = [q | k | v | output gate] and ``gates``
    fp32 [M, >= 2 H] = [input | forget] pre-activations, soft-capped by ``cap``. Per head, with ``i`` the capped input gate, ``f`` the
    log-sigmoid of the capped forget gate and a running maximum m: ``m' = max(f + m, i)``, ``S' = e^(f + m - m') S + e^(i - m') k v^T``,
    ``n'`` likewise with k alone, ``o = S'^T q / (max(|n'.q|, e^-m') + 1e-6)``, q scaled by dk^-1/2. Each head's o is RMS-normed, times
    ``norm_w`` [H dv] and the sigmoid of the output gate. ``state`` fp32 [slots, >= H (dk dv + dk + 1)]: S, n, m of all heads
    (:func:`mlstm_state_views`), zero for a new sequence, updated in place. Returns [M, H dv]."""
    if not proj.is_cuda:
        return mlstm_ref(proj, gates, norm_w, state, heads, dk, dv, cap, eps, batch, page_to_slot)
    M = proj.shape[0]
    assert proj.stride(1) == 1 and gates.stride(1) == 1 and gates.dtype == torch.float32 and norm_w.dtype == torch.float32
    assert state.is_contiguous() and state.dtype == torch.float32 and state.shape[1] >= heads * (dk * dv + dk + 1)
    out = torch.empty((M, heads * dv), dtype=proj.dtype, device=proj.device)
    if M == 0:
        return out
    batch_size = batch.block_table.shape[0]
    rows = batch.max_q_len if batch.is_prefill else batch.q_per_seq
    scratch = None
    if proj.dtype == torch.bfloat16 and proj.data_ptr() % 16 == 0 and proj.stride(0) % 8 == 0:
        size = int(lib().eredu_mlstm_scratch_bytes(heads, dk, dv, M, batch_size, rows, state.shape[1]))
        if size:
            scratch = torch.empty(size, dtype=torch.uint8, device=proj.device)
    code = lib().eredu_mlstm(ptr(proj), ptr(gates), ptr(norm_w), ptr(state), ptr(out), ptr(scratch), ptr(batch.block_table),
                             ptr(page_to_slot), ptr(batch.cu_q) if batch.is_prefill else None, ptr(batch.slots), heads, dk, dv,
                             proj.stride(0), gates.stride(0), state.shape[1], M, batch_size, batch.q_per_seq, rows,
                             batch.block_table.stride(0), 1 if proj.dtype == torch.float32 else 0, _sm_count(proj.device), cap, eps,
                             stream_ptr(proj.device))
    check(code, "eredu_mlstm")
    return out


native.register("eredu_selective_scan", I, [P] * 15 + [I] * 12 + [P])
native.register("eredu_selective_scan_scratch_elems", native.L, [I] * 6)

# Prompts of this many rows form their step sizes by a GEMM of its own in front of the scan (shorter ones and decode steps: in the scan).
SCAN_STEP_GEMM_MIN_ROWS = 64


def selective_scan_ref(x, z, params, dt_rank, dt_w, dt_b, A, D, state, batch, page_to_slot):
    c, n = A.shape
    p = params.float()
    dt = torch.nn.functional.softplus(p[:, :dt_rank] @ dt_w.float()[:, :dt_rank].t() + dt_b.float())
    Bm, Cm = p[:, dt_rank:dt_rank + n], p[:, dt_rank + n:dt_rank + 2 * n]
    xf = x.float()
    out = torch.zeros((x.shape[0], c), dtype=x.dtype, device=x.device)
    bounds = _sequences(batch)
    for b in range(len(bounds) - 1):
        r0, r1 = bounds[b], bounds[b + 1]
        if r1 <= r0 or int(batch.slots[r0]) < 0:
            continue
        cell = state[int(page_to_slot[int(batch.block_table[b, 0])])].view(-1)[:c * n].view(c, n)
        S = cell.clone()
        for t in range(r0, r1):
            S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * xf[t])[:, None] * Bm[t][None, :]
            y = (S * Cm[t][None, :]).sum(-1) + D * xf[t]
            out[t] = (y * torch.nn.functional.silu(z[t].float())).to(out.dtype)
        cell.copy_(S)
    return out


def selective_scan(x, z, params, dt_rank, dt_w, dt_b, A, D, state, batch, page_to_slot):
    """Selective scan (Mamba) over the rows of a ragged batch: per channel c and state n ``S <- exp(dt_c A[c, n]) S + dt_c x_c B_n``,
    ``y_c = sum_n S[c, n] C_n + D_c x_c``, output ``y silu(z)`` [M, channels].
    x, z [M, channels]; ``params`` [M, >= dt_rank + 2 n] = [step size input | B | C], ``dt = softplus(dt_w input + dt_b)``; dt_w [channels,
    dt_rank] in the compute dtype, dt_b, A (negative) [channels, n], D fp32; ``state`` fp32 [slots, >= channels n], in place."""
    if not x.is_cuda:
        return selective_scan_ref(x, z, params, dt_rank, dt_w, dt_b, A, D, state, batch, page_to_slot)
    from .core import linear

    c, n = A.shape
    M = x.shape[0]
    assert x.is_contiguous() and z.stride(1) == 1 and params.stride(1) == 1 and dt_w.is_contiguous() and dt_w.shape == (c, dt_rank)
    assert A.is_contiguous() and state.is_contiguous() and all(t.dtype == torch.float32 for t in (A, D, dt_b, state))
    out = torch.empty((M, c), dtype=x.dtype, device=x.device)
    if M == 0:
        return out
    B = batch.block_table.shape[0]
    rows = batch.max_q_len if batch.is_prefill else batch.q_per_seq
    dt = linear(params[:, :dt_rank], dt_w, out_dtype=torch.float32) if M >= SCAN_STEP_GEMM_MIN_ROWS and (batch.is_prefill or x.dtype == torch.float32) else None
    elems = int(lib().eredu_selective_scan_scratch_elems(c, n, B, rows, _sm_count(x.device), 1 if x.dtype == torch.float32 else 0)) if dt is not None else 0
    scratch = torch.empty(elems, dtype=torch.float32, device=x.device) if elems else None
    code = lib().eredu_selective_scan(
        ptr(x), ptr(z), ptr(params), ptr(dt), ptr(dt_w), ptr(dt_b), ptr(A), ptr(D), ptr(state), ptr(out), ptr(scratch), ptr(batch.block_table),
        ptr(page_to_slot), ptr(batch.cu_q) if batch.is_prefill else None, ptr(batch.slots), c, n, dt_rank, z.stride(0), params.stride(0),
        state[0].numel(), B, batch.q_per_seq, rows, batch.block_table.stride(0), 1 if x.dtype == torch.float32 else 0,
        _sm_count(x.device), stream_ptr(x.device))
    check(code, "eredu_selective_scan")
    return out


native.register("eredu_general_delta", I, [P] * 12 + [I] * 10 + [F, F, P])
native.register("eredu_general_delta_scratch_bytes", native.L, [I] * 7)

DELTA_UNIT_EPS = 1e-6        # added to the squared length of a key before it is made a unit vector


def general_delta_scan_ref(r, k, v, decay, rate, state):
    """r, k, decay, rate [T, H, dk], v [T, H, dv], state [H, dk, dv] (fp32). Returns (o [T, H, dv], state)."""
    u = k / torch.sqrt(k.square().sum(-1, keepdim=True) + DELTA_UNIT_EPS)
    S, out = state.clone(), []
    for t in range(r.shape[0]):
        recalled = torch.einsum("hd,hdv->hv", u[t], S)
        S = decay[t][:, :, None] * S - (rate[t] * u[t])[:, :, None] * recalled[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hd,hdv->hv", r[t], S))
    return torch.stack(out), S


def general_delta_ref(proj, w2, w0, rate_b, norm_w, state, heads, dk, dv, log_decay, eps, batch, page_to_slot):
    M, qk, vw = proj.shape[0], heads * dk, heads * dv
    x = proj.float()
    r, k, v, g, a, low = torch.split(x[:, :3 * qk + 2 * vw + w2.shape[1]], [qk, qk, vw, vw, qk, w2.shape[1]], 1)
    decay = torch.exp(-log_decay * torch.sigmoid(torch.tanh(low) @ w2.t() + w0)).view(M, heads, dk)
    rate = torch.sigmoid(a + rate_b).view(M, heads, dk)
    r, k, v = r.view(M, heads, dk), k.view(M, heads, dk), v.view(M, heads, dv)
    out = torch.zeros((M, vw), dtype=proj.dtype, device=proj.device)
    bounds = _sequences(batch)
    for b in range(len(bounds) - 1):
        r0, r1 = bounds[b], bounds[b + 1]
        if r1 <= r0 or int(batch.slots[r0]) < 0:
            continue
        slot = int(page_to_slot[int(batch.block_table[b, 0])])
        o, state[slot] = general_delta_scan_ref(r[r0:r1], k[r0:r1], v[r0:r1], decay[r0:r1], rate[r0:r1], state[slot])
        o = (o * torch.rsqrt(o.square().mean(-1, keepdim=True) + eps)).reshape(r1 - r0, vw) * norm_w
        out[r0:r1] = (o * torch.sigmoid(g[r0:r1])).to(out.dtype)
    return out


def general_delta(proj, w2, w0, rate_b, norm_w, state, heads, dk, dv, log_decay, eps, batch, page_to_slot):
    """Generalised delta rule over ``proj`` [M, >= 3 H dk + 2 H dv + rank] = [r | k | v | output gate | removal rate | decay input]. Per
    head, with the unit key u = k / |k|: ``S <- diag(w) S - (a u) (u^T S) + k v^T`` (both terms read the old state), ``o = S^T r``; decay
    ``w = exp(-log_decay sigmoid(w2 tanh(input) + w0))`` and removal rate ``a = sigmoid(rate + rate_b)`` per head and key channel. Each
    head's o is RMS-normed, times ``norm_w`` [H dv] and the sigmoid of the output gate. w2 fp32 [H dk, rank]; ``state`` fp32
    [slots, H, dk, dv], in place. Returns [M, H dv]."""
    if not proj.is_cuda:
        return general_delta_ref(proj, w2, w0, rate_b, norm_w, state, heads, dk, dv, log_decay, eps, batch, page_to_slot)
    M, rank = proj.shape[0], w2.shape[1]
    assert proj.stride(1) == 1 and state.is_contiguous() and w2.is_contiguous()
    assert all(t.dtype == torch.float32 for t in (w2, w0, rate_b, norm_w, state))
    out = torch.empty((M, heads * dv), dtype=proj.dtype, device=proj.device)
    if M == 0:
        return out
    B = batch.block_table.shape[0]
    rows = batch.max_q_len if batch.is_prefill else batch.q_per_seq
    scratch = None
    if proj.dtype == torch.bfloat16 and proj.data_ptr() % 16 == 0 and proj.stride(0) % 8 == 0 and rank % 8 == 0:
        size = int(lib().eredu_general_delta_scratch_bytes(heads, dk, dv, rank, M, B, rows))
        if size:
            scratch = torch.empty(size, dtype=torch.uint8, device=proj.device)
    code = lib().eredu_general_delta(
        ptr(proj), ptr(w2), ptr(w0), ptr(rate_b), ptr(norm_w), ptr(state), ptr(out), ptr(scratch), ptr(batch.block_table), ptr(page_to_slot),
        ptr(batch.cu_q) if batch.is_prefill else None, ptr(batch.slots), heads, dk, dv, rank, proj.stride(0), B, batch.q_per_seq, rows,
        batch.block_table.stride(0), 1 if proj.dtype == torch.float32 else 0, log_decay, eps,
        stream_ptr(proj.device))
    check(code, "eredu_general_delta")
    return out
