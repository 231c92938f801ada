"""Decoder-block operators.

Each operator has two implementations with identical semantics:

* ``*_ref`` - plain PyTorch, any device/dtype; the numerics oracle for tests and the execution path for
  CPU tensors (the fp32 CPU slice of the framework).
* the sm_100a kernel from ``liberedu_cuda.so`` for CUDA bf16 tensors. There is no fallback from the
  kernel to PyTorch on a GPU: a missing library raises.
"""
from __future__ import annotations

from os import environ as _environ

import math
from dataclasses import dataclass

import torch
import torch.nn.functional as F

from . import native
from .native import check, lib, ptr, status_word, stream_ptr

PAGE = 16


def _sm_count(device) -> int:
    return torch.cuda.get_device_properties(device).multi_processor_count


# ------------------------------------------------------------------------------------------ linear
@dataclass(frozen=True)
class XIELU:
    """xIELU (Huang, Schlag: "Deriving Activation Functions Using Integration"): ``above z^2 + z / 2`` for z > 0 and
    ``below (e^z - 1 - z) + z / 2`` elsewhere."""
    above: float
    below: float

    @classmethod
    def from_checkpoint(cls, p: float, q: float) -> "XIELU":
        """The two learned numbers behind a softplus, the lower one from 1/2 on."""
        softplus = lambda t: max(t, 0.0) + math.log1p(math.exp(-abs(t)))                # noqa: E731
        return cls(softplus(p), 0.5 + softplus(q))

    def __call__(self, z):
        n = z.clamp_max(0)
        return torch.where(z > 0, self.above * z * z, self.below * (torch.expm1(n) - n)) + z / 2


def linear_ref(x, w, bias=None, residual=None, out_dtype=None, activation=None):
    y = F.linear(x.float(), w.float(), None if bias is None else bias.float())
    if activation == "relu2":
        y = torch.relu(y).square()
    elif activation is not None:
        y = activation(y)
    if residual is not None:
        y = y + residual.float()
    return y.to(out_dtype or x.dtype)


def gated_linear_ref(x, w_gate_up, inter, bias=None, out_dtype=None, activation="silu"):
    """act(x Wg^T) * (x Wu^T) with Wg = w[:inter], Wu = w[inter:2*inter]."""
    y = F.linear(x.float(), w_gate_up.float(), None if bias is None else bias.float())
    act = torch.relu if activation == "relu" else F.silu
    return (act(y[..., :inter]) * y[..., inter:]).to(out_dtype or x.dtype)


def _norm_args(x, row_ssq, norm_eps, want_ssq, n_out):
    """(ssq_in ptr, parts, eps, dim, ssq_out tensor) for the RMSNorm fusion of the GEMM epilogue."""
    ssq_out = None
    if want_ssq:
        ssq_out = torch.empty((x.shape[0], (n_out + 127) // 128), dtype=torch.float32, device=x.device)
    if row_ssq is None:
        return None, 0, 0.0, 0, ssq_out
    assert row_ssq.dtype == torch.float32 and row_ssq.is_contiguous() and row_ssq.shape[0] == x.shape[0]
    return row_ssq, row_ssq.shape[1], float(norm_eps), x.shape[1], ssq_out


def linear(x, w, bias=None, residual=None, out_dtype=None, out=None, force_split=0, row_ssq=None, norm_eps=0.0,
           want_ssq=False, dynamic_weight=False, activation=None):
    """y = x @ w.T (+ bias) (+ residual). x: [M, K], w: [N, K].

    ``row_ssq`` ([M, parts] fp32 partial sums of squares of x's rows): the output rows are scaled by
    ``rsqrt(sum(row_ssq) / K + norm_eps)`` - an RMSNorm whose weight vector was folded into ``w``.
    ``want_ssq``: also return per-128-column-tile sums of squares of the stored output ([M, ceil(N/128)]).
    ``dynamic_weight``: ``w`` was written by a kernel enqueued just before this call (e.g. a dequantised scratch
    matrix); the kernel then does not fetch weight tiles ahead of its stream dependency.
    ``activation``: None, "relu2" (the square of ReLU) or an :class:`XIELU`, applied in the epilogue before the residual.
    fp32 operands are multiplied in true 32-bit; bf16 operands whose rows a TMA descriptor cannot describe (a row pitch or
    start that is not a multiple of 16 bytes) take the same CUDA-core kernel."""
    xielu = activation if isinstance(activation, XIELU) else None
    if activation not in (None, "relu2") and xielu is None:
        raise ValueError(f"unknown activation {activation!r}")
    if not x.is_cuda:
        if row_ssq is not None:
            x = x.float() * torch.rsqrt(row_ssq.sum(-1, keepdim=True) / x.shape[1] + norm_eps)
        y = linear_ref(x, w, bias, residual, out_dtype or w.dtype, activation)
        return (y, y.float().pow(2).sum(-1, keepdim=True)) if want_ssq else y
    if x.dtype == torch.float32 or not (_tma_rows(x) and _tma_rows(w)):
        assert residual is None and row_ssq is None and not want_ssq, "the CUDA-core linear has no norm or residual fusion"
        return _linear_simt(x, w, bias, out_dtype or x.dtype, activation, out)
    assert x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16, "CUDA linear is bf16"
    M, K = x.shape
    N = w.shape[0]
    out_dtype = out_dtype or torch.bfloat16
    assert out_dtype in (torch.bfloat16, torch.float32)
    assert x.stride(1) == 1 and w.stride(1) == 1
    if out is None:
        out = torch.empty((M, N), dtype=out_dtype, device=x.device)
    ssq_in, parts, eps, dim, ssq_out = _norm_args(x, row_ssq, norm_eps, want_ssq, N)
    if M == 0:
        return (out, ssq_out) if want_ssq else out
    code = lib().eredu_gemm_bf16(
        ptr(x), ptr(w), ptr(out), ptr(residual), ptr(bias), M, N, K, x.stride(0), w.stride(0), out.stride(0),
        residual.stride(0) if residual is not None else 0, w.shape[0], 0, 0, 1 if out_dtype == torch.float32 else 0,
        force_split, _sm_count(x.device), ptr(status_word(x.device)), ptr(ssq_in), parts, eps, dim, ptr(ssq_out),
        (1 if dynamic_weight else 0) | (2 if activation == "relu2" else 8 if xielu else 0), xielu.above if xielu else 0.0,
        xielu.below if xielu else 0.0, stream_ptr(x.device))
    check(code, "eredu_gemm_bf16")
    return (out, ssq_out) if want_ssq else out


def _tma_rows(t) -> bool:
    return t.stride(1) == 1 and (t.stride(0) * t.element_size()) % 16 == 0 and t.data_ptr() % 16 == 0


native.register("eredu_gemm_simt", native.I, [native.P] * 4 + [native.I] * 9 + [native.F, native.F, native.P])


def _linear_simt(x, w, bias, out_dtype, activation, out=None):
    """fp32-accumulating GEMM on the CUDA cores: fp32 operands, or bf16 operands of any pitch."""
    assert x.dtype == w.dtype and x.dtype in (torch.float32, torch.bfloat16) and x.stride(1) == 1 and w.stride(1) == 1
    assert bias is None or (bias.dtype == x.dtype and bias.is_contiguous())
    M, K = x.shape
    xielu = isinstance(activation, XIELU)
    act = 4 if xielu else {None: 0, "relu2": 1, "gated_silu": 2, "gated_relu": 3}[activation]
    N = w.shape[0] // 2 if act in (2, 3) else w.shape[0]
    if out is None:
        out = torch.empty((M, N), dtype=out_dtype, device=x.device)
    if M == 0:
        return out
    code = lib().eredu_gemm_simt(ptr(x), ptr(w), ptr(out), ptr(bias), M, N, K, x.stride(0), w.stride(0), out.stride(0),
                                 1 if x.dtype == torch.float32 else 0, 1 if out.dtype == torch.float32 else 0,
                                 act, activation.above if xielu else 0.0, activation.below if xielu else 0.0, stream_ptr(x.device))
    check(code, "eredu_gemm_simt")
    return out


def gated_linear(x, w_gate_up, inter, bias=None, out=None, force_split=0, row_ssq=None, norm_eps=0.0, activation="silu"):
    """Fused gated up-projection (SwiGLU; ``activation`` "relu": ReLU of the gate): one GEMM kernel, activation applied in the
    epilogue (``row_ssq``: see linear). fp32 operands, and bf16 rows a TMA descriptor cannot describe, take the CUDA-core kernel."""
    if activation not in ("silu", "relu"):
        raise ValueError(f"unknown activation {activation!r}")
    if not x.is_cuda:
        if row_ssq is not None:
            x = x.float() * torch.rsqrt(row_ssq.sum(-1, keepdim=True) / x.shape[1] + norm_eps)
        return gated_linear_ref(x, w_gate_up, inter, bias, w_gate_up.dtype, activation)
    if x.dtype == torch.float32 or not (_tma_rows(x) and _tma_rows(w_gate_up)):
        assert row_ssq is None, "the CUDA-core linear has no norm fusion"
        return _linear_simt(x, w_gate_up, bias, x.dtype, "gated_" + activation, out)
    assert x.dtype == torch.bfloat16 and w_gate_up.dtype == torch.bfloat16
    M, K = x.shape
    if out is None:
        out = torch.empty((M, inter), dtype=torch.bfloat16, device=x.device)
    if M == 0:
        return out
    ssq_in, parts, eps, dim, _ = _norm_args(x, row_ssq, norm_eps, False, inter)
    code = lib().eredu_gemm_bf16(
        ptr(x), ptr(w_gate_up), ptr(out), None, ptr(bias), M, inter, K, x.stride(0), w_gate_up.stride(0),
        out.stride(0), 0, w_gate_up.shape[0], 1, inter, 0, force_split, _sm_count(x.device),
        ptr(status_word(x.device)), ptr(ssq_in), parts, eps, dim, None, 4 if activation == "relu" else 0, 0.0, 0.0, stream_ptr(x.device))
    check(code, "eredu_gemm_bf16(dual)")
    return out


# ------------------------------------------------------------------------------------------ norm
def rmsnorm_ref(x, weight, eps, residual=None, weight_offset=0.0):
    h = x.float()
    if residual is not None:
        h = (h + residual.float()).to(x.dtype).float()
    y = h * torch.rsqrt(h.pow(2).mean(-1, keepdim=True) + eps) * (weight.float() + weight_offset)
    return y.to(x.dtype), (h.to(x.dtype) if residual is not None else None)


def rmsnorm(x, weight, eps, residual=None, weight_offset=0.0):
    """Returns (normed, h) where h = x + residual (None when no residual was given)."""
    if not x.is_cuda:
        return rmsnorm_ref(x, weight, eps, residual, weight_offset)
    assert x.dtype == torch.bfloat16 and weight.dtype == torch.float32 and x.is_contiguous()
    M, H = x.shape
    y = torch.empty_like(x)
    h = torch.empty_like(x) if residual is not None else None
    code = lib().eredu_rmsnorm(ptr(x), ptr(residual), ptr(weight), ptr(y), ptr(h), M, H, eps, weight_offset,
                               stream_ptr(x.device))
    check(code, "eredu_rmsnorm")
    return y, h


native.register("eredu_rms_residual", native.I, [native.P] * 5 + [native.I] * 4 + [native.F, native.P])
native.register("eredu_embedding_stream", native.I, [native.P] * 6 + [native.I] * 4 + [native.F, native.P])
native.register("eredu_rms_routed_residual", native.I, [native.P] * 13 + [native.I] * 8 + [native.F, native.P])
native.register("eredu_qkv_prepare", native.I, [native.P] * 9 + [native.I] * 10 + [native.F, native.P])


MAX_ROUTES = 32         # routes of a token the kernels add up


def rms_residual_ref(y, weight, eps, residual=None, act_dtype=None, routed=None, conv=None, want_act=True):
    n = y.float() if y is not None else 0.0
    if routed is not None:
        n = n + routed.summed()
    n = n * torch.rsqrt(n.square().mean(-1, keepdim=True) + eps) * weight.float()
    if residual is not None:
        n = residual + n
    if not want_act:
        return n, None
    if conv is not None:
        from .conv import stream_conv_ref

        return n, stream_conv_ref(n, conv, act_dtype or y.dtype)
    return n, n.to(act_dtype or y.dtype)


def rms_residual(y, weight, eps, residual=None, act_dtype=None, routed=None, conv=None, want_act=True):
    """Norm on a sublayer's output: ``x = residual + weight * y / rms(y)`` in fp32, and its copy in ``act_dtype``.
    ``weight``: fp32, one number for all coordinates ([1]) or one per coordinate. Without a residual only the copy of the
    normalised rows is made (the first result is then None, or the copy itself when it is fp32). Returns (x, copy).
    ``routed`` (:class:`ops.moe.RoutedRows`): expert rows whose weighted sum is added to ``y`` (which may be None) first.
    ``conv`` (:class:`ops.conv.StreamConv`; decode steps of one token per sequence): the copy is ``x + conv(x)``.
    ``want_act=False``: no copy."""
    act_dtype = act_dtype or y.dtype
    ref = y if y is not None else routed.rows
    if not ref.is_cuda:
        return rms_residual_ref(y, weight, eps, residual, act_dtype, routed, conv, want_act)
    M, W = y.shape if y is not None else (routed.weights.shape[0], routed.rows.shape[1])
    assert (y is None or y.is_contiguous()) and weight.dtype == torch.float32 and weight.numel() in (1, W)
    assert residual is None or (residual.dtype == torch.float32 and residual.is_contiguous())
    act = torch.empty((M, W), dtype=act_dtype, device=ref.device) if want_act else None
    fp32 = ref.dtype == torch.float32
    if routed is None and conv is None:
        shared = want_act and act_dtype == torch.float32
        x = act if shared else (torch.empty((M, W), dtype=torch.float32, device=ref.device) if residual is not None else None)
        code = lib().eredu_rms_residual(ptr(y), ptr(weight), ptr(residual), ptr(x), None if shared else ptr(act), M, W,
                                        1 if fp32 else 0, 0 if weight.numel() == 1 else 1, eps, stream_ptr(ref.device))
        check(code, "eredu_rms_residual")
        return x, act
    assert residual is not None and weight.numel() == W and act_dtype == ref.dtype
    x = torch.empty((M, W), dtype=torch.float32, device=ref.device)
    rows = pos = w = None
    k = 0
    if routed is not None and routed.weights.shape[1] > MAX_ROUTES:
        y, routed = (routed.summed() if y is None else y.float() + routed.summed()).to(ref.dtype), None
    if routed is not None:
        rows, pos, w = routed.rows, routed.route_pos, routed.weights
        k = w.shape[1]
        assert rows.is_contiguous() and rows.shape[1] == W and w.shape[0] == M and w.dtype == torch.float32 and (y is None or y.dtype == rows.dtype)
    taps = state = table = p2s = slots = None
    if conv is not None:
        assert want_act and not conv.batch.is_prefill and conv.batch.q_per_seq == 1
        taps, state = conv.checked(W)
        if state is not None:
            table, p2s, slots = conv.batch.block_table, conv.page_to_slot, conv.batch.slots
    code = lib().eredu_rms_routed_residual(
        ptr(y), ptr(rows), ptr(pos), ptr(w), ptr(weight), ptr(residual), ptr(x), ptr(act), ptr(taps), ptr(state), ptr(table), ptr(p2s), ptr(slots),
        M, W, k, taps.shape[0] if taps is not None else 0, state[0].numel() if state is not None else 0,
        table.stride(0) if table is not None else 0, 1 if fp32 else 0, 1 if W % 4 == 0 else 0, eps, stream_ptr(ref.device))
    check(code, "eredu_rms_routed_residual")
    return x, act


def embedding_stream(ids, table, scale=1.0, want_act=True, positions=None, inv_freq=None):
    """Rows of ``table`` times ``scale`` as the start of an fp32 residual stream: (fp32 rows, rows in the table's dtype or None).
    With ``inv_freq`` (fp32, one per pair of columns) sinusoidal position vectors are added: column 2 i gets
    sin(position * inv_freq[i]), column 2 i + 1 the cosine."""
    if not table.is_cuda:
        x = table[ids.long()].float() * scale
        if inv_freq is not None:
            a = positions.float()[:, None] * inv_freq.float()[None]
            x = x + torch.stack((a.sin(), a.cos()), -1).flatten(1)[:, :x.shape[1]]
        return x, (x.to(table.dtype) if want_act else None)
    assert ids.dtype == torch.int32 and table.is_contiguous()
    M, W = ids.shape[0], table.shape[1]
    assert inv_freq is None or (inv_freq.dtype == torch.float32 and inv_freq.numel() == (W + 1) // 2 and positions.dtype == torch.int32)
    x = torch.empty((M, W), dtype=torch.float32, device=table.device)
    fp32 = table.dtype == torch.float32
    act = x if fp32 else (torch.empty((M, W), dtype=table.dtype, device=table.device) if want_act else None)
    code = lib().eredu_embedding_stream(ptr(ids), ptr(table), ptr(x), None if fp32 else ptr(act), ptr(positions) if inv_freq is not None else None,
                                        ptr(inv_freq), M, W, table.shape[0], 1 if fp32 else 0, scale, stream_ptr(table.device))
    check(code, "eredu_embedding_stream")
    return x, act


native.register("eredu_residual_norm", native.I, [native.P] * 9 + [native.I] * 6 + [native.F, native.P])


def residual_norm_ref(x, y=None, routed=None, weight=None, bias=None, eps=1e-5, act_dtype=None, center=True):
    out = x.float()
    if y is not None:
        out = out + y.float()
    if routed is not None:
        out = out + routed.summed()
    if weight is None:
        return out, None
    n = out - out.mean(-1, keepdim=True) if center else out
    n = n * torch.rsqrt(n.square().mean(-1, keepdim=True) + eps) * weight.float()
    return out, (n if bias is None else n + bias.float()).to(act_dtype or x.dtype)


def residual_norm(x, y=None, routed=None, weight=None, bias=None, eps=1e-5, act_dtype=None, center=True):
    """What a layer's sublayers add to the fp32 stream and the norm of the sum in front of the next layer, in one launch:
    ``x' = x + y + sum_k w_k rows_k`` with a sublayer's output ``y`` and the expert rows of ``routed`` (:class:`ops.moe.RoutedRows`)
    in the compute dtype, both optional; ``act = weight * (x' - mean) / sqrt(var + eps) + bias`` in ``act_dtype`` (``center=False``:
    RMSNorm; ``bias`` optional; no ``weight``: no norm). Returns (x', act); x' is x itself when nothing is added."""
    if not x.is_cuda:
        return residual_norm_ref(x, y, routed, weight, bias, eps, act_dtype, center)
    M, W = x.shape
    act_dtype = act_dtype or torch.bfloat16
    assert x.dtype == torch.float32 and x.is_contiguous() and act_dtype in (torch.bfloat16, torch.float32)
    assert y is None or (y.dtype == act_dtype and y.is_contiguous() and y.shape == x.shape)
    assert weight is None or (weight.dtype == torch.float32 and weight.numel() == W)
    assert bias is None or (bias.dtype == torch.float32 and bias.numel() == W)
    rows = pos = w = None
    k = 0
    if routed is not None:
        rows, pos, w = routed.rows, routed.route_pos, routed.weights
        k = w.shape[1]
        assert rows.dtype == act_dtype and rows.is_contiguous() and rows.shape[1] == W and w.shape[0] == M and w.dtype == torch.float32
    adds = y is not None or routed is not None
    out = torch.empty_like(x) if adds else x
    act = torch.empty((M, W), dtype=act_dtype, device=x.device) if weight is not None else None
    if M == 0 or (not adds and weight is None):
        return out, act
    code = lib().eredu_residual_norm(ptr(x), ptr(y), ptr(rows), ptr(pos), ptr(w), ptr(weight), ptr(bias), ptr(out) if adds else None,
                                     ptr(act), M, W, k, 1 if act_dtype == torch.float32 else 0, 1 if center else 0,
                                     1 if W % 4 == 0 else 0, eps, stream_ptr(x.device))
    check(code, "eredu_residual_norm")
    return out, act


native.register("eredu_branch_norm", native.I, [native.P] * 9 + [native.I] * 4 + [native.F, native.F, native.P])


def branch_norm_ref(x, branches, weight, next_weight=None, eps=1e-5, act_dtype=None, branch_weights=None, gain=1.0):
    def rms(t, w):
        t = t.float()
        return t * torch.rsqrt(t.square().mean(-1, keepdim=True) + eps) * w.float()

    y = sum(b.float() if branch_weights is None else rms(b, w) for b, w in zip(branches, branch_weights or branches)) * gain
    out = x + rms(y, weight)
    return out, None if next_weight is None else rms(out, next_weight).to(act_dtype or x.dtype)


def branch_norm(x, branches, weight, next_weight=None, eps=1e-5, act_dtype=None, branch_weights=None, gain=1.0):
    """A norm behind a sublayer, the residual sum and the norm in front of the next one, in one launch:
    ``x' = x + rms(gain * sum_j y_j) * weight``, ``act = rms(x') * next_weight`` in ``act_dtype`` (None without a next weight). One or
    two ``branches`` y_j in the compute dtype; with ``branch_weights`` each is RMS-normed with its own weight before the sum. x fp32.
    Returns (x', act)."""
    if not x.is_cuda:
        return branch_norm_ref(x, branches, weight, next_weight, eps, act_dtype, branch_weights, gain)
    M, W = x.shape
    act_dtype = act_dtype or torch.bfloat16
    assert x.dtype == torch.float32 and x.is_contiguous() and 1 <= len(branches) <= 2
    assert all(y.is_contiguous() and y.dtype == act_dtype and y.shape == x.shape for y in branches)
    ws = list(branch_weights) if branch_weights is not None else [None] * len(branches)
    assert len(ws) == len(branches) and all(w is None or (w.dtype == torch.float32 and w.numel() == W) for w in (*ws, weight, next_weight))
    out = torch.empty_like(x)
    act = torch.empty((M, W), dtype=act_dtype, device=x.device) if next_weight is not None else None
    if M == 0:
        return out, act
    second = len(branches) == 2
    code = lib().eredu_branch_norm(ptr(x), ptr(branches[0]), ptr(branches[1]) if second else None, ptr(ws[0]), ptr(ws[1]) if second else None,
                                   ptr(weight), ptr(next_weight), ptr(out), ptr(act), M, W, 1 if act_dtype == torch.float32 else 0,
                                   1 if W % 4 == 0 else 0, gain, eps, stream_ptr(x.device))
    check(code, "eredu_branch_norm")
    return out, act


# ------------------------------------------------------------------------------------------ rope + kv append
def qkv_prepare_ref(qkv, positions, slots, inv_freq, k_cache, v_cache, n_q, n_kv, dk, dv, q_norm_w=None, k_norm_w=None,
                    norm_eps=1e-6, value_norm=False, append=True):
    M = qkv.shape[0]
    rot = 2 * inv_freq.shape[0]
    ang = positions.float()[:, None] * inv_freq.float()[None, :]
    cos, sin = ang.cos()[:, None, :], ang.sin()[:, None, :]

    def rms(t):
        return t * torch.rsqrt(t.square().mean(-1, keepdim=True) + norm_eps)

    def project(t, w, heads):
        if w is not None:
            t = rms(t) * w.float()
        t = t.view(M, heads, dk)
        u, v = t[..., :rot // 2], t[..., rot // 2:rot]
        return torch.cat((u * cos - v * sin, v * cos + u * sin, t[..., rot:]), -1)

    x = qkv.float()
    if append:
        k = project(x[:, n_q * dk:(n_q + n_kv) * dk], k_norm_w, n_kv)
        v = x[:, (n_q + n_kv) * dk:(n_q + n_kv) * dk + n_kv * dv].reshape(M, n_kv, dv)
        v = rms(v) if value_norm else v
        ok = slots >= 0
        page, off = slots[ok] // PAGE, slots[ok] % PAGE
        k_cache[page, :, off] = k[ok].to(k_cache.dtype)
        v_cache[page, :, off] = v[ok].to(v_cache.dtype)
    return project(x[:, :n_q * dk], q_norm_w, n_q).to(qkv.dtype).contiguous()


def qkv_prepare(qkv, positions, slots, inv_freq, k_cache, v_cache, n_q, n_kv, dk, dv, q_norm_w=None, k_norm_w=None,
                norm_eps=1e-6, value_norm=False, append=True):
    """``qkv`` [M, n_q dk (+ n_kv dk + n_kv dv)]: RMSNorm over the WHOLE query and the whole key projection (weights of that
    size; None: no norm), rotation of the first ``2 len(inv_freq)`` dims of every head (pairs i, i + half), optional
    weight-free RMSNorm of every value head, keys and values scattered into their pages. ``append=False``: the rows hold
    queries only (the layer reads another layer's pages). Returns q [M, n_q, dk] in qkv's dtype."""
    if not qkv.is_cuda:
        return qkv_prepare_ref(qkv, positions, slots, inv_freq, k_cache, v_cache, n_q, n_kv, dk, dv, q_norm_w, k_norm_w,
                               norm_eps, value_norm, append)
    assert positions.dtype == torch.int32 and slots.dtype == torch.int64 and inv_freq.dtype == torch.float32
    assert qkv.stride(1) == 1 and k_cache.is_contiguous() and v_cache.is_contiguous() and k_cache.dtype == qkv.dtype
    M = qkv.shape[0]
    q = torch.empty((M, n_q, dk), dtype=qkv.dtype, device=qkv.device)
    code = lib().eredu_qkv_prepare(ptr(qkv), ptr(q), ptr(k_cache), ptr(v_cache), ptr(positions), ptr(slots), ptr(inv_freq),
                                   ptr(q_norm_w), ptr(k_norm_w), M, qkv.stride(0), n_q, n_kv, dk, dv, 2 * inv_freq.shape[0],
                                   1 if value_norm else 0, 1 if append else 0, 1 if qkv.dtype == torch.float32 else 0,
                                   norm_eps, stream_ptr(qkv.device))
    check(code, "eredu_qkv_prepare")
    return q


def rope_kv_ref(qkv, positions, slots, inv_freq, k_cache, v_cache, n_q, n_kv, head_dim, rot=None, interleaved=False,
                attn_factor=1.0, q_norm_w=None, k_norm_w=None, norm_eps=1e-6, norm_w_off=0.0, mrope_section=None):
    """``positions`` [M], or [3, M] (temporal, height, width axes of multimodal prompts) with ``mrope_section``: frequency
    index f then takes its angle from axis f % 3 while f < 3 * section[axis] (interleaved T H W T H W ... layout), the
    temporal axis otherwise."""
    M = qkv.shape[0]
    D = head_dim
    rot = rot or D
    x = qkv.float().view(M, n_q + 2 * n_kv, D)
    q, k, v = x[:, :n_q], x[:, n_q:n_q + n_kv], x[:, n_q + n_kv:]

    def hnorm(t, w):
        if w is None:
            return t
        y = t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + norm_eps) * (w.float() + norm_w_off)
        return y.to(qkv.dtype).float()

    q, k = hnorm(q, q_norm_w), hnorm(k, k_norm_w)
    if positions.dim() == 2:
        axes = positions.float()[:, :, None] * inv_freq.float()[None, None, :]          # [3, M, rot/2]
        ang = axes[0].clone()
        for axis, offset in ((1, 1), (2, 2)):
            idx = slice(offset, int(mrope_section[axis]) * 3, 3)
            ang[:, idx] = axes[axis][:, idx]
    else:
        ang = positions.float()[:, None] * inv_freq.float()[None, :]  # [M, rot/2]
    cos, sin = (ang.cos() * attn_factor)[:, None, :], (ang.sin() * attn_factor)[:, None, :]

    def rotate(t):
        tr, tp = t[..., :rot], t[..., rot:]
        if interleaved:
            a, b = tr[..., 0::2], tr[..., 1::2]
            out = torch.stack((a * cos - b * sin, b * cos + a * sin), dim=-1).flatten(-2)
        else:
            a, b = tr[..., : rot // 2], tr[..., rot // 2:]
            out = torch.cat((a * cos - b * sin, b * cos + a * sin), dim=-1)
        return torch.cat((out, tp), dim=-1)

    q, k = rotate(q), rotate(k)
    ok = slots >= 0
    page, off = (slots[ok] // PAGE), (slots[ok] % PAGE)
    k_cache[page, :, off] = k[ok].to(k_cache.dtype)
    v_cache[page, :, off] = v[ok].to(v_cache.dtype)
    return q.to(qkv.dtype).contiguous()


def rope_kv(qkv, positions, slots, inv_freq, k_cache, v_cache, n_q, n_kv, head_dim, rot=None, interleaved=False,
            attn_factor=1.0, q_norm_w=None, k_norm_w=None, norm_eps=1e-6, norm_w_off=0.0, q_out=None, mrope_section=None):
    """Per-head q/k norm (optional) + RoPE on q and k, K/V scattered into their cache pages. Returns q [M,n_q,D].
    Three-axis positions ([3, M], prompts with images) take the tensor-operation path on either device."""
    if not qkv.is_cuda or head_dim not in KERNEL_HEAD_DIMS or positions.dim() == 2:
        return rope_kv_ref(qkv, positions, slots, inv_freq, k_cache, v_cache, n_q, n_kv, head_dim, rot, interleaved,
                           attn_factor, q_norm_w, k_norm_w, norm_eps, norm_w_off, mrope_section)
    M = qkv.shape[0]
    rot = rot or head_dim
    assert positions.dtype == torch.int32 and slots.dtype == torch.int64 and inv_freq.dtype == torch.float32
    if q_out is None:
        q_out = torch.empty((M, n_q, head_dim), dtype=qkv.dtype, device=qkv.device)
    code = lib().eredu_rope_kv(ptr(qkv), ptr(q_out), ptr(k_cache), ptr(v_cache), ptr(positions), ptr(slots),
                               ptr(inv_freq), ptr(q_norm_w), ptr(k_norm_w), M, qkv.stride(0), n_q, n_kv, head_dim, rot,
                               1 if interleaved else 0, attn_factor, norm_eps, norm_w_off, stream_ptr(qkv.device))
    check(code, "eredu_rope_kv")
    return q_out


# Head sizes the attention and RoPE kernels are instantiated for; other sizes (256 in the Qwen3-Next family) run through
# the tensor-operation references on either device, which read lengths on the host: such models decode eagerly.
KERNEL_HEAD_DIMS = (64, 128)


# ------------------------------------------------------------------------------------------ attention
def _gather_kv(cache, block_table_row, kv_len):
    n_pages = (kv_len + PAGE - 1) // PAGE
    pages = cache[block_table_row[:n_pages].long()]  # [n_pages, n_kv, 16, D]
    return pages.permute(1, 0, 2, 3).reshape(cache.shape[1], n_pages * PAGE, cache.shape[3])[:, :kv_len]


def attention_ref(q, k_cache, v_cache, block_table, seq_lens, q_lens, scale, window=0, sinks=None, bidir=None, chunk=0):
    """q: [total_q, n_q, D]; the last q_lens[b] positions of sequence b are its queries (causal).
    ``chunk``: a query sees the keys of its own chunk of positions [c * chunk, (c + 1) * chunk) only.
    ``bidir``: per sequence None or an int tensor [kv_len] of group ids (negative: none); positions of one group see each
    other in both directions, whatever the causal order and the window say (soft tokens of one image)."""
    total, n_q, D = q.shape
    n_kv = k_cache.shape[1]
    group = n_q // n_kv
    out = torch.empty((total, n_q, v_cache.shape[3]), dtype=q.dtype, device=q.device)
    start = 0
    for b, (kv_len, ql) in enumerate(zip(seq_lens.tolist(), q_lens)):
        k = _gather_kv(k_cache, block_table[b], kv_len).float()  # [n_kv, T, D]
        v = _gather_kv(v_cache, block_table[b], kv_len).float()
        qb = q[start:start + ql].float().permute(1, 0, 2)  # [n_q, ql, D]
        k = k.repeat_interleave(group, dim=0)
        v = v.repeat_interleave(group, dim=0)
        s = torch.einsum("hqd,hkd->hqk", qb, k) * scale
        qpos = torch.arange(kv_len - ql, kv_len, device=q.device)[:, None]
        kpos = torch.arange(kv_len, device=q.device)[None, :]
        mask = kpos <= qpos
        if window > 0:
            mask = mask & (kpos > qpos - window)
        if chunk > 0:
            mask = mask & (kpos // chunk == qpos // chunk)
        if bidir is not None and bidir[b] is not None:
            grp = bidir[b].to(q.device)
            mask = mask | ((grp[kv_len - ql:kv_len, None] == grp[None, :kv_len]) & (grp[kv_len - ql:kv_len, None] >= 0))
        s = s.masked_fill(~mask[None], float("-inf"))
        if sinks is not None:
            s = torch.cat((s, sinks.float()[:, None, None].expand(n_q, ql, 1)), dim=-1)
            p = torch.softmax(s, dim=-1)[..., :-1]
        else:
            p = torch.softmax(s, dim=-1)
        out[start:start + ql] = torch.einsum("hqk,hkd->hqd", p, v).permute(1, 0, 2).to(q.dtype)
        start += ql
    return out


TC_PREFILL = _environ.get("EREDU_TC_PREFILL", "1") != "0"      # head size 64 / 128: the tcgen05 kernel (else the mma.sync one)


native.register("eredu_attn_simt", native.I, [native.P] * 8 + [native.I] * 12 + [native.F, native.P])


def _attention_simt(q, k_cache, v_cache, block_table, seq_lens, cu_q, q_per_seq, max_q_len, scale, window, chunk, sinks):
    """Paged attention on the CUDA cores: fp32 caches, and head sizes the tensor-core kernels are not built for."""
    assert q.is_contiguous() and k_cache.is_contiguous() and v_cache.is_contiguous() and q.dtype == k_cache.dtype == v_cache.dtype
    out = torch.empty((q.shape[0], q.shape[1], v_cache.shape[3]), dtype=q.dtype, device=q.device)
    if q.shape[0] == 0:
        return out
    code = lib().eredu_attn_simt(ptr(q), ptr(k_cache), ptr(v_cache), ptr(out), ptr(block_table), ptr(seq_lens), ptr(cu_q),
                                 ptr(sinks), seq_lens.shape[0], q_per_seq, max_q_len, block_table.stride(0), q.shape[1],
                                 k_cache.shape[1], q.shape[2], v_cache.shape[3], v_cache.shape[3], int(window), int(chunk),
                                 1 if q.dtype == torch.float32 else 0, scale, stream_ptr(q.device))
    check(code, "eredu_attn_simt")
    return out


def _tensor_core_dims(q, k_cache, v_cache) -> bool:
    """Head sizes (multiples of 8 up to 128, keys and values may differ) and dtype of the tensor-core attention kernels."""
    dk, dv = q.shape[2], v_cache.shape[3]
    return (q.dtype == torch.bfloat16 and dk % 8 == 0 and dv % 8 == 0 and 0 < dk <= 128 and 0 < dv <= 128
            and k_cache.is_contiguous() and v_cache.is_contiguous())


def attention_prefill(q, k_cache, v_cache, block_table, seq_lens, cu_q, max_q_len, scale, window=0, sinks=None,
                      out=None, chunk=0):
    """``window`` > 0: a query at position p sees keys in (p - window, p]; ``chunk`` > 0: the keys of its own chunk of
    positions. Key and value widths are those of the caches. Returns [total_q, n_q, value width]."""
    if q.is_cuda and (chunk > 0 or q.dtype == torch.float32 or v_cache.shape[3] != q.shape[2]):
        if not _tensor_core_dims(q, k_cache, v_cache):
            return _attention_simt(q, k_cache, v_cache, block_table, seq_lens, cu_q, 0, max_q_len, scale, window, chunk, sinks)
    elif not q.is_cuda or q.shape[2] not in KERNEL_HEAD_DIMS:
        q_lens = (cu_q[1:] - cu_q[:-1]).tolist()
        return attention_ref(q, k_cache, v_cache, block_table, seq_lens, q_lens, scale, window, sinks, chunk=chunk)
    assert q.dtype == torch.bfloat16 and q.is_contiguous()
    assert block_table.dtype == torch.int32 and seq_lens.dtype == torch.int32 and cu_q.dtype == torch.int32
    dk, dv = q.shape[2], v_cache.shape[3]
    if out is None:
        out = torch.empty((q.shape[0], q.shape[1], dv), dtype=q.dtype, device=q.device)
    B = seq_lens.shape[0]
    only_tc = chunk > 0 or dk != dv
    if ((TC_PREFILL or only_tc) and (only_tc or dk in (64, 128)) and k_cache.is_contiguous() and v_cache.is_contiguous()
            and k_cache.shape[2] == 16 and k_cache.shape[3] == dk and v_cache.shape[:3] == k_cache.shape[:3] and out.is_contiguous()
            and (sinks is None or (sinks.dtype == torch.float32 and sinks.is_contiguous()))):
        # tcgen05 kernel (csrc/kernels/attention_tc.cu): QK^T and PV on the 5th-generation tensor cores, pages by TMA
        code = lib().eredu_attn_prefill_tc(ptr(q), ptr(k_cache), ptr(v_cache), ptr(out), ptr(block_table), ptr(seq_lens),
                                           ptr(cu_q), ptr(sinks), B, q.shape[0], max_q_len, block_table.stride(0),
                                           k_cache.shape[0], q.shape[1], k_cache.shape[1], dk, dv, int(window), int(chunk), scale,
                                           ptr(status_word(q.device)), stream_ptr(q.device))
        check(code, "eredu_attn_prefill_tc")
        return out
    code = lib().eredu_attn_prefill(ptr(q), ptr(k_cache), ptr(v_cache), ptr(out), ptr(block_table), ptr(seq_lens),
                                    ptr(cu_q), ptr(sinks), B, max_q_len, block_table.stride(0), q.shape[1],
                                    k_cache.shape[1], q.shape[2], window, scale, stream_ptr(q.device))
    check(code, "eredu_attn_prefill")
    return out


import os as _os

_SPLIT_WAVES = int(_os.environ.get("EREDU_DECODE_SPLIT_WAVES", "2"))   # CTAs per SM the split-KV grid aims for


CLUSTER_SPLITS = 8      # splits the decode kernel combines through distributed shared memory (portable cluster size)
FUSED_ROPE_MAX_NEW = 8  # new tokens per sequence the fused RoPE + append decode path takes


def decode_splits(batch, n_kv, max_kv_len, sm_count=148):
    """Split-KV factor: enough CTAs to fill the GPU once (a second wave costs more than it returns: the CTAs of the
    following kernel are already resident under programmatic dependent launch), at least 8 pages per split."""
    ctas = max(1, batch * n_kv)
    pages = max(1, (max_kv_len + PAGE - 1) // PAGE)
    want = max(1, (_SPLIT_WAVES * sm_count) // ctas)
    splits = int(max(1, min(want, pages // 8 if pages >= 8 else 1, 32)))
    # up to CLUSTER_SPLITS splits combine inside a thread-block cluster (no scratch, no second pass over global memory):
    # prefer that form while a split then still has at most 32 pages (8 per warp)
    if splits > CLUSTER_SPLITS and pages <= 32 * CLUSTER_SPLITS:
        splits = CLUSTER_SPLITS
    return splits


def attention_decode(q, k_cache, v_cache, block_table, seq_lens, q_per_seq, scale, splits=1, window=0, sinks=None,
                     scratch=None, out=None, chunk=0):
    """q: [B * q_per_seq, n_q, D]; ``window`` / ``chunk`` as in :func:`attention_prefill`. ``scratch`` = (part_o, part_ml, counters) from :func:`decode_scratch` when
    splits > 1 (fp32 partials and zeroed int32 arrival tickets)."""
    if q.is_cuda and (chunk > 0 or q.dtype == torch.float32 or v_cache.shape[3] != q.shape[2]):
        if not _tensor_core_dims(q, k_cache, v_cache) or q.shape[1] // k_cache.shape[1] > 32:
            return _attention_simt(q, k_cache, v_cache, block_table, seq_lens, None, q_per_seq, q_per_seq, scale, window, chunk,
                                   sinks)
    elif not q.is_cuda or q.shape[2] not in KERNEL_HEAD_DIMS:
        return attention_ref(q, k_cache, v_cache, block_table, seq_lens, [q_per_seq] * seq_lens.shape[0], scale,
                             window, sinks, chunk=chunk)
    assert q.dtype == torch.bfloat16 and q.is_contiguous()
    B = seq_lens.shape[0]
    n_q, D = q.shape[1], v_cache.shape[3]
    if out is None:
        out = torch.empty((q.shape[0], n_q, D), dtype=q.dtype, device=q.device)
    part_o = part_ml = counters = None
    if splits > CLUSTER_SPLITS:
        if scratch is None:
            scratch = decode_scratch(B, q_per_seq, n_q, D, splits, q.device)
        part_o, part_ml, counters = scratch
        assert part_o.numel() >= B * q_per_seq * n_q * splits * D and part_ml.numel() >= B * q_per_seq * n_q * splits * 2
        assert counters.numel() >= B * k_cache.shape[1] and counters.dtype == torch.int32
    code = lib().eredu_attn_decode(ptr(q), ptr(k_cache), ptr(v_cache), ptr(out), ptr(block_table), ptr(seq_lens),
                                   ptr(sinks), ptr(part_o), ptr(part_ml), ptr(counters), B, q_per_seq, block_table.stride(0), n_q,
                                   k_cache.shape[1], q.shape[2], D, splits, window, chunk, scale, stream_ptr(q.device))
    check(code, "eredu_attn_decode")
    return out


def attention_decode_rope(qkv, k_cache, v_cache, block_table, seq_lens, q_per_seq, scale, positions, slots, inv_freq,
                          n_q, n_kv, head_dim, rot=None, interleaved=False, attn_factor=1.0, q_norm_w=None, k_norm_w=None,
                          norm_eps=1e-6, norm_w_off=0.0, splits=1, window=0, sinks=None, scratch=None, chunk=0, value_dim=None,
                          norm_whole=False, value_norm=False, append=True):
    """Decode attention straight from the qkv projection output [B * q_per_seq, >= (n_q + 2 n_kv) * D]: per-head
    q/k norm, RoPE and the KV append run inside the attention kernel (one launch instead of two). CPU tensors and
    head sizes without a kernel compose the two reference operators.
    ``norm_whole`` / ``value_norm`` / ``append``: the preparation of :func:`qkv_prepare` (norms over whole projections, value
    heads of width ``value_dim``, rows that hold queries only) instead of that of :func:`rope_kv`."""
    value_dim = value_dim or head_dim
    if norm_whole or value_norm or not append or value_dim != head_dim or chunk:
        whole = (qkv.is_cuda and qkv.dtype == torch.bfloat16 and _tma_rows(qkv) and head_dim % 8 == 0 and value_dim % 8 == 0
                 and max(head_dim, value_dim) <= 128 and n_q // n_kv <= 32 and q_per_seq <= FUSED_ROPE_MAX_NEW
                 and splits <= CLUSTER_SPLITS and norm_whole and not interleaved)
        if not whole:
            assert norm_whole and not interleaved and norm_w_off == 0.0 and attn_factor == 1.0
            q = qkv_prepare(qkv, positions, slots, inv_freq, k_cache, v_cache, n_q, n_kv, head_dim, value_dim, q_norm_w, k_norm_w,
                            norm_eps, value_norm, append)
            return attention_decode(q, k_cache, v_cache, block_table, seq_lens, q_per_seq, scale, splits, window, sinks, scratch,
                                    chunk=chunk)
        rot = 2 * inv_freq.shape[0]
    elif not qkv.is_cuda or head_dim not in KERNEL_HEAD_DIMS or positions.dim() != 1 or q_per_seq > FUSED_ROPE_MAX_NEW:
        q = rope_kv(qkv, positions, slots, inv_freq, k_cache, v_cache, n_q, n_kv, head_dim, rot, interleaved, attn_factor,
                    q_norm_w, k_norm_w, norm_eps, norm_w_off)
        return attention_decode(q, k_cache, v_cache, block_table, seq_lens, q_per_seq, scale, splits, window, sinks, scratch)
    assert qkv.dtype == torch.bfloat16 and qkv.stride(1) == 1
    assert positions.dtype == torch.int32 and slots.dtype == torch.int64 and inv_freq.dtype == torch.float32
    B = seq_lens.shape[0]
    out = torch.empty((qkv.shape[0], n_q, value_dim), dtype=qkv.dtype, device=qkv.device)
    part_o = part_ml = counters = None
    if splits > CLUSTER_SPLITS:
        if scratch is None:
            scratch = decode_scratch(B, q_per_seq, n_q, head_dim, splits, qkv.device)
        part_o, part_ml, counters = scratch
        assert part_o.numel() >= B * q_per_seq * n_q * splits * head_dim and counters.numel() >= B * n_kv
    code = lib().eredu_attn_decode_rope(ptr(qkv), qkv.stride(0), ptr(k_cache), ptr(v_cache), ptr(out), ptr(block_table),
                                        ptr(seq_lens), ptr(sinks), ptr(part_o), ptr(part_ml), ptr(counters), ptr(positions),
                                        ptr(slots), ptr(inv_freq), ptr(q_norm_w), ptr(k_norm_w), B, q_per_seq,
                                        block_table.stride(0), n_q, n_kv, head_dim, value_dim,
                                        head_dim if rot is None else rot, 1 if interleaved else 0, splits, window, chunk,
                                        int(norm_whole), int(value_norm), int(append), scale, attn_factor, norm_eps,
                                        norm_w_off, stream_ptr(qkv.device))
    check(code, "eredu_attn_decode_rope")
    return out


def decode_scratch(batch, q_per_seq, n_q, head_dim, splits, device):
    rows = batch * q_per_seq * n_q
    return (torch.empty(rows * splits * head_dim, dtype=torch.float32, device=device),
            torch.empty(rows * splits * 2, dtype=torch.float32, device=device),
            torch.zeros(batch * n_q, dtype=torch.int32, device=device))


# ------------------------------------------------------------------------------------------ embedding / activation
def embedding(ids, table, vocab_start=0, scale=1.0, want_ssq=False):
    """Rows of ``table`` for ``ids`` (zero rows for ids outside this shard). ``want_ssq``: also the per-row sum of
    squares ([M, 1] fp32) consumed by a GEMM with a folded RMSNorm."""
    if not table.is_cuda:
        local = ids.long() - vocab_start
        ok = (local >= 0) & (local < table.shape[0])
        out = table[local.clamp(0, table.shape[0] - 1)] * ok[:, None].to(table.dtype)
        out = out * scale if scale != 1.0 else out
        return (out, out.float().pow(2).sum(-1, keepdim=True)) if want_ssq else out
    assert ids.dtype == torch.int32 and table.dtype == torch.bfloat16
    M, H = ids.shape[0], table.shape[1]
    out = torch.empty((M, H), dtype=table.dtype, device=table.device)
    ssq = torch.empty((M, 1), dtype=torch.float32, device=table.device) if want_ssq else None
    code = lib().eredu_embedding(ptr(ids), ptr(table), ptr(out), M, H, vocab_start, table.shape[0], scale, ptr(ssq),
                                 stream_ptr(table.device))
    check(code, "eredu_embedding")
    return (out, ssq) if want_ssq else out


def silu_mul(x, inter, limit=0.0):
    """x: [M, 2*inter] = [gate | up] -> silu(gate) * up."""
    if not x.is_cuda:
        g, u = x[..., :inter].float(), x[..., inter:].float()
        if limit > 0:
            g, u = g.clamp(max=limit), u.clamp(-limit, limit)
        return (F.silu(g) * u).to(x.dtype)
    M = x.shape[0]
    y = torch.empty((M, inter), dtype=x.dtype, device=x.device)
    code = lib().eredu_silu_mul(ptr(x), ptr(y), M, inter, x.stride(0), limit, stream_ptr(x.device))
    check(code, "eredu_silu_mul")
    return y
