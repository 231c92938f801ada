"""Gulazen at sizes that resemble a real model's layers, beside the framework's closest model at equal size (Qwen3-MoE with a sliding
window: the same widths, attention geometry, experts and shared experts, dense layers of as many parameters), and its kernels beside the
like kernels of that and the other families, each against its roofline.

    python -m benchmarks.bench_gulazen [--sizes small medium large] [--no-kernels] [--no-models]
    python bench.py --design gulazen

Timing as in bench_nidozen: models by CUDA events around ``Engine.prefill`` and around replays of the captured decode step; kernels as
captured graphs of launches over separate buffers that together exceed L2.
"""
from __future__ import annotations

import argparse
import json

import torch

from eredu_b200 import ops
from eredu_b200.models.config import ModelConfig
from eredu_b200.ops import moe as moe_ops
from eredu_b200.ops import native

from . import bench_nidozen as B
from .bench_nidozen import BF, DEV, F32, batch_of, rnd

# width, pairs of layers (dense, routed), query heads, kv heads, head size, dense ff, experts, top, expert ff, shared ff
SIZES = {"small": (1024, 8, 16, 4, 64, 4096, 32, 4, 512, 1024), "medium": (2048, 8, 16, 4, 128, 8192, 64, 6, 768, 1536),
         "large": (4096, 8, 32, 8, 128, 16384, 64, 6, 1536, 3072)}
WINDOW, KEEP, TAPS, CAP = 1024, 64, 4, 30.0
VOCAB = 32000
SFU_PER_CLOCK = 16 * 148          # exponentials, reciprocals a clock
SM_GHZ = 1.965


def gulazen_config(size: str) -> ModelConfig:
    W, n, H, G, D, ff, E, top, eff, shared = SIZES[size]
    at = {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "mask": {"size": WINDOW, "keep_first": KEEP}, "scale": D ** -0.5, "softcap": CAP}
    moe = {"kind": "moe", "expert": {"ff": eff}, "router": {"experts": E, "top": top}, "shared": {"ff": shared}}
    layers = [{"type": "attention", "mixer": at, "mlp": {"kind": "dense", "ff": ff}}, {"type": "attention", "mixer": at, "mlp": moe}] * n
    return ModelConfig.from_hf_dict({"architecture": "Gulazen", "width": W, "vocab": VOCAB, "norm": {"eps": 1e-6}, "canon": {"taps": TAPS},
                                     "layers": layers})


def closest_config(size: str) -> ModelConfig:
    W, n, H, G, D, ff, E, top, eff, shared = SIZES[size]
    return ModelConfig.from_hf_dict({
        "model_type": "qwen3_moe", "hidden_size": W, "num_hidden_layers": 2 * n, "num_attention_heads": H, "num_key_value_heads": G, "head_dim": D,
        "intermediate_size": (ff * 2 // 3 + 63) // 64 * 64, "vocab_size": VOCAB, "num_experts": E, "num_experts_per_tok": top, "decoder_sparse_step": 2,
        "moe_intermediate_size": eff, "shared_expert_intermediate_size": shared, "norm_topk_prob": True, "tie_word_embeddings": True,
        "sliding_window": WINDOW, "use_sliding_window": True, "max_position_embeddings": 65536, "rms_norm_eps": 1e-6})


def random_model(cfg: ModelConfig):
    """Random weights drawn on the device."""
    from eredu_b200.models.llama import _shape_of, build_from_tensors, build_random
    from eredu_b200.models.moe import make_moe_factory

    if cfg.model_type == "gulazen":
        return build_random(cfg, DEV, BF, seed=0)
    W, s = cfg.hidden_size, cfg.shared_expert_intermediate_size
    shared = {"gate_proj": (s, W), "up_proj": (s, W), "down_proj": (W, s)}

    def shape(name):
        if ".mlp.shared_expert." in name and cfg.layer_is_moe(int(name.split(".")[2])):
            return shared.get(name.split(".")[-2])
        return _shape_of(cfg, name)

    def get(name):
        n = shape(name)
        return torch.ones(n, device=DEV) if name.endswith("norm.weight") else torch.randn(n, device=DEV, dtype=BF) * 0.02

    return build_from_tensors(cfg, get, lambda name: shape(name) is not None, DEV, BF, moe_factory=make_moe_factory())


# ---------------------------------------------------------------------------------------------- kernels
def kernel_numbers(size: str, T: int = 8192, Bn: int = 32, context: int = 2048, only: str = "") -> list:
    W, _, H, G, D, ff, E, top, eff, shared = SIZES[size]
    bw, tf = B.peaks()
    rows = []

    def add(name, nbytes, flops, make, like=None, like_make=None, like_bytes=None, like_flops=None, sfu=0, like_sfu=0):
        """``sfu``: exponentials and reciprocals."""
        if only and only not in name:
            return
        us = B.per_launch_us(make, nbytes)
        roof = lambda b, f, s: max(b / bw / 1e3, f / tf / 1e6, s / SFU_PER_CLOCK / SM_GHZ / 1e3)      # noqa: E731
        r = roof(nbytes, flops, sfu)
        entry = {"kernel": name, "us": round(us, 2), "roofline_us": round(r, 2), "x": round(us / r, 2)}
        if like_make is not None:
            lb, lf = like_bytes or nbytes, like_flops if like_flops is not None else flops
            lus = B.per_launch_us(like_make, lb)
            lr = roof(lb, lf, like_sfu)
            entry.update(like=like, like_us=round(lus, 2), like_roofline_us=round(lr, 2), like_x=round(lus / lr, 2), relative=round(us / r / (lus / lr), 2))
        rows.append(entry)
        print(json.dumps(entry), flush=True)

    ones = torch.ones(W, device=DEV)
    taps = rnd(TAPS, W, dt=F32, s=0.2)
    talk = (torch.eye(H, device=DEV) + torch.randn(H, H, device=DEV) * 0.05).to(BF)
    sinks = torch.zeros(H, device=DEV)
    for phase, M in (("prefill", T), ("decode", Bn)):
        prefill = phase == "prefill"
        bt = batch_of(T, 1, T, True) if prefill else batch_of(1, Bn, context, False)
        bt.sm_count = 148
        if not prefill:
            bt.max_kv_len = context
        pages = int(bt.block_table.max()) + 1
        seqs = bt.block_table.shape[0]
        p2s = torch.zeros(pages, dtype=torch.int32, device=DEV)
        p2s[bt.block_table[:, 0].long()] = torch.arange(seqs, device=DEV, dtype=torch.int32)

        # ---- the stream
        def conv_of(state):
            return ops.StreamConv(taps, state, bt, p2s)

        def norm(i):
            x, y = rnd(M, W, dt=F32), rnd(M, W)
            return lambda: ops.rms_residual(y, ones, 1e-6, residual=x, act_dtype=BF)

        def norm_conv(i):
            x, y, s = rnd(M, W, dt=F32), rnd(M, W), rnd(seqs, (TAPS - 1) * W, dt=F32)
            return lambda: ops.rms_residual(y, ones, 1e-6, residual=x, act_dtype=BF, conv=conv_of(s))

        ids = torch.stack([torch.randperm(E, device=DEV)[:top] for _ in range(M)]).int() if M <= 64 else torch.rand(M, E, device=DEV).topk(top, -1).indices.int()
        plan = moe_ops.ExpertPlan(ids, top, 0, E, 16, M * top)
        wts = torch.rand(M, top, device=DEV)

        def norm_routed(i):
            x, y, r = rnd(M, W, dt=F32), rnd(M, W), rnd(M * top, W)
            routed = moe_ops.RoutedRows(r, plan.route_pos, wts)
            return lambda: ops.rms_residual(y, ones, 1e-6, residual=x, act_dtype=BF, routed=routed)

        def like_routed(i):
            x, y, r = rnd(M, W, dt=F32), rnd(M, W), rnd(M * top, W)
            routed = moe_ops.RoutedRows(r, plan.route_pos, wts)
            return lambda: ops.residual_norm(x, y, routed, ones, None, 1e-6, BF, center=False)

        add(f"{phase} norm behind {top} expert rows and the shared expert", M * W * (12 + 2 * top), 0, norm_routed, "residual_norm of the same rows", like_routed)
        if prefill:
            def conv(i):
                x, s = rnd(M, W, dt=F32), rnd(seqs, (TAPS - 1) * W, dt=F32)
                return lambda: ops.stream_conv(x, conv_of(s), BF)

            def like_conv(i):
                x, s = rnd(M, W), torch.zeros(pages, TAPS - 1, W, device=DEV, dtype=BF)
                w = rnd(W, TAPS, dt=F32)
                return lambda: ops.short_conv(x, w, None, s, bt.block_table, bt.cu_q, 1, bt.positions, bt.slots, M, mode=1)

            add("prefill stream_conv", M * W * 6, 0, conv, "short_conv of as many channels, bf16", like_conv, M * W * 4)
        else:
            add("decode norm, residual and convolution", M * W * (12 + 8 * (TAPS - 1)), 0, norm_conv, "rms_residual (norm, residual, copy)", norm, M * W * 12)
        table, tok, freq = rnd(VOCAB, W), torch.randint(0, VOCAB, (M,), device=DEV, dtype=torch.int32), torch.rand(W // 2, device=DEV)

        def embed(i, with_positions=True):
            return lambda: ops.embedding_stream(tok, table, want_act=False, positions=bt.positions, inv_freq=freq if with_positions else None)

        add(f"{phase} embedding and position vectors", M * W * 6, 0, embed, "embedding_stream", lambda i: embed(i, False))

        # ---- routing
        def route(i, scoring="topk_softmax"):
            z, x = rnd(M, E, dt=F32), rnd(M, W)
            if prefill:
                return lambda: moe_ops.route(z, top, scoring, False)
            return lambda: moe_ops.route_plan_gather(z, x, top, scoring, False, 1.0, None, 0, E)

        add(f"{phase} routing, softmax of the chosen" + ("" if prefill else ", plan and gather"), M * (E * 4 + top * 8) if prefill else M * (E * 4 + W * 2 + top * (8 + 2 * W)), 0, route,
            "routing by sigmoids", lambda i: route(i, "sigmoid"))

        # ---- xIELU
        def up(i, act=ops.XIELU(0.8, 1.1)):
            x, w = rnd(M, W), rnd(ff, W, s=0.02)
            return lambda: ops.linear(x, w, activation=act)

        add(f"{phase} projection with xIELU", (M * (W + ff) + ff * W) * 2, 2 * M * W * ff, up, "the same with squared ReLU", lambda i: up(i, "relu2"))

        # ---- attention
        seen = min(WINDOW + KEEP, context)
        pairs = WINDOW * T - WINDOW * WINDOW / 2 + KEEP * (T - WINDOW) if prefill else Bn * seen
        like_pairs = WINDOW * T - WINDOW * WINDOW / 2 if prefill else Bn * WINDOW

        def attn(i):
            q, kc, vc = rnd(M, H, D), rnd(pages, G, 16, D), rnd(pages, G, 16, D)
            return lambda: ops.talking_attention(q, kc, vc, bt, talk, D ** -0.5, CAP, sinks, WINDOW, KEEP)

        def like_attn(i):
            q, kc, vc = rnd(M, H, D), rnd(pages, G, 16, D), rnd(pages, G, 16, D)
            if prefill:
                return lambda: ops.attention_prefill(q, kc, vc, bt.block_table, bt.seq_lens, bt.cu_q, T, D ** -0.5, window=WINDOW, sinks=sinks)
            sp = ops.decode_splits(Bn, G, WINDOW)
            return lambda: ops.attention_decode(q, kc, vc, bt.block_table, bt.seq_lens, 1, D ** -0.5, splits=sp, window=WINDOW, sinks=sinks)

        io = M * H * D * 4 + (T * G * D * 4 if prefill else Bn * seen * G * D * 4)
        add(f"{phase} attention, heads mixed, capped", io, pairs * H * (4 * D + 2 * H), attn, "attention, same window, sinks", like_attn,
            M * H * D * 4 + (T if prefill else Bn * WINDOW) * G * D * 4, 4 * like_pairs * H * D, sfu=3 * pairs * H, like_sfu=like_pairs * H)
    native.check_status(DEV)
    return rows


def run(sizes, steps: int, models: bool = True, kernels: bool = True, closest: bool = True) -> dict:
    torch.cuda.set_device(DEV)
    result = {"models": {}, "kernels": {}}
    for size in sizes:
        if models:
            entry = {"gulazen": B.model_numbers(gulazen_config(size), steps, build=random_model)}
            if closest:
                entry["qwen3_moe"] = B.model_numbers(closest_config(size), min(steps, 8), build=random_model)
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
