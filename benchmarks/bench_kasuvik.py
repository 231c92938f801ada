"""Kasuvik at sizes that resemble a real model's layers, beside the framework's closest model at equal size (Nemotron-H: the same widths,
attention geometry and feed-forward weights, Mamba-2 blocks in the place of the scan and of the delta rule), and its kernels beside the
like kernels of that and the other families, each against its roofline.

    python -m benchmarks.bench_kasuvik [--sizes small medium large] [--no-kernels] [--no-models]
    python bench.py --design kasuvik

Timing as in bench_nidozen: models by CUDA events around ``Engine.prefill`` and around replays of the captured decode step; kernels as
captured graphs of launches over separate buffers that together exceed L2.
"""
from __future__ import annotations

import argparse
import json

import torch

from eredu_b200 import ops
from eredu_b200.models.config import ModelConfig
from eredu_b200.ops import native

from . import bench_nidozen as B
from .bench_nidozen import BF, DEV, F32, batch_of, rnd

# width, pairs of layers, query heads, kv heads, head size, scan channels, states, step size rank, delta heads, delta head size
SIZES = {"small": (1024, 8, 16, 4, 64, 2048, 16, 64, 16, 64), "medium": (2048, 8, 16, 4, 128, 4096, 16, 128, 32, 64),
         "large": (4096, 8, 32, 8, 128, 8192, 16, 256, 32, 128)}
WINDOW, POOL, TAPS, SCAN_TAPS = 1024, 16, 3, 4
VOCAB = 32000
DELTA_RANK = 16


def kasuvik_config(size: str) -> ModelConfig:
    W, n, H, G, D, C, N, R, DH, DD = SIZES[size]
    mlp = {"kind": "dense", "ff": 2 * W}
    left = {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "conv": TAPS, "mask": {"size": WINDOW, "pool": POOL}, "rot": {"dims": D, "base": 10000.0},
            "scale": D ** -0.5}
    layers = [{"type": "parallel", "mixer": {"left": left, "right": {"inner": C, "state": N, "dt_rank": R, "conv": SCAN_TAPS}}, "mlp": mlp},
              {"type": "general_delta", "mixer": {"heads": DH, "dim": DD}, "mlp": mlp}] * n
    return ModelConfig.from_hf_dict({"architecture": "Kasuvik", "width": W, "vocab": VOCAB, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0},
                                     "layers": layers})


def closest_config(size: str) -> ModelConfig:
    W, n, H, G, D, C, N, R, DH, DD = SIZES[size]
    return ModelConfig.from_hf_dict({
        "model_type": "nemotron_h", "hybrid_override_pattern": "*M-M-" * n, "hidden_size": W, "num_attention_heads": H, "num_key_value_heads": G,
        "head_dim": D, "mamba_num_heads": C // 64, "mamba_head_dim": 64, "ssm_state_size": 64, "n_groups": 8, "conv_kernel": SCAN_TAPS,
        "intermediate_size": 3 * W, "vocab_size": VOCAB, "n_routed_experts": 0, "layer_norm_epsilon": 1e-5, "max_position_embeddings": 65536})


# ---------------------------------------------------------------------------------------------- kernels
def kernel_numbers(size: str, T: int = 8192, Bn: int = 32, context: int = 2048, only: str = "") -> list:
    W, _, H, G, D, C, N, R, DH, DD = SIZES[size]
    bw, tf = B.peaks()
    rows = []

    def add(name, nbytes, flops, make, like=None, like_make=None, like_bytes=None, like_flops=None):
        if only and only not in name:
            return
        us = B.per_launch_us(make, nbytes)
        roof = max(nbytes / bw / 1e3, flops / tf / 1e6)
        entry = {"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "x": round(us / roof, 2)}
        if like_make is not None:
            lb, lf = like_bytes or nbytes, like_flops if like_flops is not None else flops
            lus = B.per_launch_us(like_make, lb)
            lroof = max(lb / bw / 1e3, lf / tf / 1e6)
            entry.update(like=like, like_us=round(lus, 2), like_roofline_us=round(lroof, 2), like_x=round(lus / lroof, 2),
                         relative=round(us / roof / (lus / lroof), 2))
        rows.append(entry)
        print(json.dumps(entry), flush=True)

    lib, P_ = native.lib(), native.ptr
    ones = torch.ones(W, device=DEV)
    inv = torch.rand(D // 2, device=DEV)
    qkv = (H + 2 * G) * D
    cols = qkv + 2 * C
    for phase, M in (("prefill", T), ("decode", Bn)):
        prefill = phase == "prefill"
        n, ctx = (1, T) if prefill else (Bn, context)
        bt = batch_of(M // n, n, ctx, prefill)
        bt.portions = [(0, T)]
        pages = int(bt.block_table.max()) + 1
        p2s = torch.zeros(pages, dtype=torch.int32, device=DEV)
        p2s[bt.block_table[:, 0].long()] = torch.arange(n, device=DEV, dtype=torch.int32)
        cache = lambda: (rnd(pages, G, 16, D), rnd(pages, G, 16, D))                    # noqa: E731
        means = lambda: tuple(rnd(pages, G, -(-16 // POOL), D) for _ in range(2))       # noqa: E731

        # ---- norms around a sublayer, beside the norm + fp32 residual of a sublayer's output
        def two(i):
            x, a, b = rnd(M, W, dt=F32), rnd(M, W), rnd(M, W)
            return lambda: ops.branch_norm(x, [a, b], ones, ones, 1e-5, BF, (ones, ones), 0.5)

        def one(i):
            x, a = rnd(M, W, dt=F32), rnd(M, W)
            return lambda: ops.branch_norm(x, [a], ones, ones, 1e-5, BF)

        def like_norm(i):
            x, y = rnd(M, W, dt=F32), rnd(M, W)
            return lambda: ops.rms_residual(y, ones, 1e-5, residual=x, act_dtype=BF)

        add(f"{phase} branch_norm, two branches", M * W * 14, 0, two, "rms_residual (norm, residual, copy)", like_norm, M * W * 12)
        add(f"{phase} branch_norm, one branch", M * W * 12, 0, one, "rms_residual (norm, residual, copy)", like_norm, M * W * 12)

        # ---- gated projection
        def relu(act):
            def make(i):
                x, w = rnd(M, W), rnd(4 * W, W, s=0.02)
                return lambda: ops.gated_linear(x, w, 2 * W, activation=act)
            return make

        add(f"{phase} gated projection, ReLU", 4 * W * W * 2 + M * 3 * W * 2, 8.0 * M * W * W, relu("relu"), "the same with SiLU", relu("silu"))

        # ---- convolutions, rotation, append
        ht, ct, cb, temp = rnd(TAPS, qkv, dt=F32), rnd(SCAN_TAPS, C, dt=F32), rnd(C, dt=F32), torch.ones(H, device=DEV)
        hist = (TAPS - 1) * qkv

        def conv(i):
            x, (kc, vc), st = rnd(M, cols), cache(), torch.zeros(n, hist + (SCAN_TAPS - 1) * C, device=DEV)
            heads = ops.ConvHeads(ht, H, G, D, D, inv, kc, vc, temp, POOL, means(), 0)
            chans = ops.ConvChannels(ct, cb, qkv, hist)
            return lambda: ops.conv_project(x, st, bt, p2s, heads, chans)

        qw, kw = torch.ones(H * D, device=DEV), torch.ones(G * D, device=DEV)
        ct8 = ct.t().contiguous()

        def like_conv(i):
            x, z, (kc, vc) = rnd(M, qkv), rnd(M, 2 * C), cache()
            st = torch.zeros(pages, SCAN_TAPS - 1, C, device=DEV, dtype=BF)

            def run():
                ops.qkv_prepare(x, bt.positions, bt.slots, inv, kc, vc, H, G, D, D, qw, kw, 1e-5)
                ops.short_conv(z, ct8, cb, st, bt.block_table, bt.cu_q, bt.q_per_seq, bt.positions, bt.slots, bt.max_q_len, 1, 0)
            return run

        history = 0 if prefill else n * (hist + (SCAN_TAPS - 1) * C) * 8
        add(f"{phase} conv_project", M * (qkv + C) * 4 + history, 0, conv, "qkv_prepare, then short_conv", like_conv, M * (qkv + C) * 4 + (0 if prefill else n * 3 * C * 4))

        # ---- attention over a window and the blocks behind it
        if prefill:
            tokens = WINDOW * T - WINDOW * WINDOW / 2
            pairs = tokens + sum(max(0, (i - WINDOW + 1) // POOL) for i in range(T))

            def pool(i):
                (kc, vc), m = cache(), means()
                return lambda: ops.pool_blocks(kc, vc, m, bt, POOL)

            add("prefill pool_blocks", T * G * D * 4 + T // POOL * G * D * 8, 0, pool)

            def attn(i):
                q, (kc, vc), m = rnd(M, H, D), cache(), means()
                return lambda: ops.pooled_attention(q, kc, vc, m, bt, D ** -0.5, WINDOW, POOL)

            def window(i):
                q, (kc, vc) = rnd(M, H, D), cache()
                return lambda: ops.attention_prefill(q, kc, vc, bt.block_table, bt.seq_lens, bt.cu_q, T, D ** -0.5, window=WINDOW)

            io = T * (2 * H + 2 * G) * D * 2
            add("prefill attention, window and blocks (with pool_blocks)", io, 4 * pairs * H * D, attn, "attention, same window", window, io, 4 * tokens * H * D)
        else:
            seen = min(WINDOW, context)
            blocks = (context - WINDOW) // POOL

            def attn(i):
                q, (kc, vc), m = rnd(M, H, D), cache(), means()
                return lambda: ops.pooled_attention(q, kc, vc, m, bt, D ** -0.5, WINDOW, POOL)

            def window(i):
                q, (kc, vc) = rnd(M, H, D), cache()
                sp = ops.decode_splits(Bn, G, WINDOW)
                return lambda: ops.attention_decode(q, kc, vc, bt.block_table, bt.seq_lens, 1, D ** -0.5, splits=sp, window=WINDOW)

            add("decode attention, window and blocks", Bn * (seen + blocks) * G * D * 4, 4.0 * Bn * H * (seen + blocks) * D, attn, "attention, same window", window,
                Bn * seen * G * D * 4, 4.0 * Bn * H * seen * D)

        # ---- selective scan (with its step size projection), beside the closest model's scan
        cut = -(-(R + 2 * N) // 8) * 8
        A, Dk, tb = -torch.rand(C, N, device=DEV) * 8 - 0.5, torch.ones(C, device=DEV), torch.full((C,), -4.0, device=DEV)

        def scan(i):
            x, p, z, w = rnd(M, C), rnd(M, cut), rnd(M, cols), rnd(C, R, s=0.05)
            st = torch.zeros(n, C * N, device=DEV)
            return lambda: ops.selective_scan(x, z[:, qkv + C:], p, R, w, tb, A, Dk, st, bt, p2s)

        MH = C // 64

        def mamba2(i):
            x, b, c = rnd(n, M // n, MH, 64), rnd(n, M // n, 8, 64, s=0.2), rnd(n, M // n, 8, 64, s=0.2)
            dt, a, d = torch.rand(n, M // n, MH, device=DEV) * 0.1, -torch.rand(MH, device=DEV), torch.ones(MH, device=DEV)
            s, o = torch.zeros(n, MH, 64, 64, device=DEV), torch.empty(n, M // n, MH, 64, device=DEV, dtype=BF)
            if prefill:                                        # what the closest model runs on long prompts
                return lambda: ops.mamba2_scan(x, b, c, dt, a, d, s)
            return lambda: lib.eredu_mamba2_scan(*map(P_, (x, b, c, dt, a, d, s, o)), n, M // n, MH, 8, 64, 64, native.stream_ptr(DEV))

        def mingru(i):
            x, s = rnd(M, 3 * C), torch.zeros(n, C, device=DEV)
            return lambda: ops.mingru_scan(x, s, C, bt, p2s)

        io = M * (C * 6 + (R + 2 * N) * 2) + C * R * 2 + n * C * N * 8
        mio = M * (C * 4 + 16 * 64 * 2 + MH * 4) + n * MH * 64 * 64 * 8
        add(f"{phase} selective_scan (step sizes, scan, gate)", io, 2.0 * M * C * R, scan, "mamba2_scan (closest model)", mamba2, mio, 4.0 * M * MH * 64 * 64)
        add(f"{phase} selective_scan (step sizes, scan, gate)", io, 2.0 * M * C * R, scan, "mingru_scan, equal channels", mingru, M * C * 8 + n * C * 8, 0)

        # ---- generalised delta rule, beside gated linear attention and the delta rule of other families
        qk = DH * DD
        w2, w0, rb, nw = rnd(qk, DELTA_RANK, dt=F32, s=0.2), rnd(qk, dt=F32) - 2, rnd(qk, dt=F32), torch.ones(qk, device=DEV)

        def delta(i):
            x, s = rnd(M, 5 * qk + DELTA_RANK), torch.zeros(n, DH, DD, DD, device=DEV)
            return lambda: ops.general_delta(x, w2, w0, rb, nw, s, DH, DD, DD, 0.6, 1e-5, bt, p2s)

        a2b, gnw = rnd(qk, dt=F32), torch.ones(DD, device=DEV)

        def gla(i):
            x, s = rnd(M, 4 * qk + 16), torch.zeros(n, DH, DD, DD, device=DEV)
            return lambda: ops.gla_attention(x, w2, a2b, gnw, s, DH, DD, DD, 16.0, 1e-5, bt, p2s)

        def kda(i):
            q, k, v = rnd(n, M // n, DH, DD, s=0.3), rnd(n, M // n, DH, DD, s=0.1), rnd(n, M // n, DH, DD)
            ld, be = -torch.rand(n, M // n, DH, DD, device=DEV) * 0.1, torch.rand(n, M // n, DH, device=DEV)
            s, o = torch.zeros(n, DH, DD, DD, device=DEV), torch.empty(n, M // n, DH, DD, device=DEV, dtype=BF)
            return lambda: lib.eredu_gated_delta_scan(*map(P_, (q, k, v, ld, be, s, o)), n, M // n, DH, DD, DD, 1, native.stream_ptr(DEV))

        state = n * DH * DD * DD * 8
        fl = 6.0 * M * DH * DD * DD
        add(f"{phase} general_delta (gates, recurrence, norm, output gate)", M * (6 * qk + DELTA_RANK) * 2 + state, fl, delta, "gated_delta_scan, vector decay", kda,
            M * (4 * qk * 2 + qk * 4 + DH * 4) + state, fl)
        add(f"{phase} general_delta (gates, recurrence, norm, output gate)", M * (6 * qk + DELTA_RANK) * 2 + state, fl, delta, "gla_attention, equal state", gla,
            M * (5 * qk + 16) * 2 + state, 4.0 * M * DH * DD * DD)
    native.check_status(DEV)
    return rows


def run(sizes, steps: int, models: bool = True, kernels: bool = True, closest: bool = True) -> dict:
    torch.cuda.set_device(DEV)
    result = {"models": {}, "kernels": {}}
    for size in sizes:
        if models:
            entry = {"kasuvik": B.model_numbers(kasuvik_config(size), steps)}
            if closest:
                entry["nemotron_h"] = B.model_numbers(closest_config(size), min(steps, 32))
            result["models"][size] = entry
            print(json.dumps({"size": size, **entry}), flush=True)
        if kernels:
            result["kernels"][size] = kernel_numbers(size)
    return result


def main() -> None:
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", nargs="*", default=list(SIZES), choices=list(SIZES))
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--no-models", action="store_true")
    ap.add_argument("--no-kernels", action="store_true")
    ap.add_argument("--no-closest", action="store_true", help="skip the closest model")
    ap.add_argument("--only", default="", help="kernels whose name contains this")
    a = ap.parse_args()
    if a.only:
        for size in a.sizes:
            kernel_numbers(size, only=a.only)
        return
    run(a.sizes, a.steps, not a.no_models, not a.no_kernels, not a.no_closest)


if __name__ == "__main__":
    main()
