"""Lenitar at sizes that resemble a real model's layers, beside the framework's closest model at equal size (Kimi Linear: the same
widths, latent-attention geometry, recurrent-state size and group-routed experts), and its kernels beside the like kernels of that
and the other families, each against its roofline.

    python -m benchmarks.bench_lenitar [--sizes small medium large] [--no-kernels] [--no-models]
    python bench.py --design lenitar

Timing as in bench_nidozen: models by CUDA events around ``Engine.prefill`` and around replays of the captured decode step; kernels as
captured graphs of launches over separate buffers that together exceed L2.
"""
from __future__ import annotations

import argparse
import json

import torch

from eredu_b200 import ops
from eredu_b200.models.config import ModelConfig
from eredu_b200.ops import latent as latent_ops
from eredu_b200.ops import moe as moe_ops
from eredu_b200.ops import native

from . import bench_nidozen as B
from .bench_nidozen import BF, DEV, F32, batch_of, rnd

# width, pairs of layers, heads, dim, rot, vdim, kv rank, q rank, recurrent heads, state rows, state columns, experts, top, groups, kept, ff
SIZES = {"small": (1024, 8, 16, 64, 32, 64, 256, 768, 4, 128, 256, 32, 4, 4, 2, 512),
         "medium": (2048, 8, 16, 128, 64, 128, 512, 1024, 8, 128, 256, 64, 6, 8, 4, 768),
         "large": (4096, 8, 32, 128, 64, 128, 512, 1536, 8, 256, 512, 64, 6, 8, 4, 1536)}
WINDOW = 1024
VOCAB = 32000


def lenitar_config(size: str) -> ModelConfig:
    W, n, H, D, P, V, R, Q, RH, dk, dv, E, top, G, keep, ff = SIZES[size]
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": E, "top": top, "groups": {"count": G, "keep": keep}}}
    at = {"heads": H, "dim": D, "rot_dim": P, "vdim": V, "kv_rank": R, "q_rank": Q, "mask": {"size": WINDOW}, "scale": (D + P) ** -0.5,
          "rot": {"dims": P, "base": 10000.0}}
    layers = [{"type": "latent_attention", "mixer": at, "mlp": mlp},
              {"type": "mlstm", "mixer": {"heads": RH, "dim": dk, "vdim": dv, "gate_cap": 15.0}, "mlp": mlp}] * n
    return ModelConfig.from_hf_dict({"architecture": "Lenitar", "width": W, "vocab": VOCAB, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0},
                                     "layers": layers})


def closest_config(size: str) -> ModelConfig:
    W, n, H, D, P, V, R, Q, RH, dk, dv, E, top, G, keep, ff = SIZES[size]
    return ModelConfig.from_hf_dict({
        "model_type": "kimi_linear", "hidden_size": W, "num_hidden_layers": 2 * n, "num_attention_heads": H, "num_key_value_heads": H,
        "q_lora_rank": Q, "kv_lora_rank": R, "qk_nope_head_dim": D, "qk_rope_head_dim": P, "v_head_dim": V, "intermediate_size": ff,
        "vocab_size": VOCAB, "mla_use_nope": True, "num_experts": E, "num_experts_per_token": top, "moe_intermediate_size": ff,
        "num_shared_experts": 0, "num_expert_group": G, "topk_group": keep, "use_grouped_topk": True, "moe_renormalize": False,
        "first_k_dense_replace": 0, "tie_word_embeddings": False, "max_position_embeddings": 65536, "rms_norm_eps": 1e-5,
        "linear_attn_config": {"full_attn_layers": [2 * i + 1 for i in range(n)], "kda_layers": [2 * i + 2 for i in range(n)],
                               "num_heads": RH * dk * dv // (128 * 128), "head_dim": 128, "short_conv_kernel_size": 4}})


def random_model(cfg: ModelConfig):
    """Random weights drawn on the device."""
    from eredu_b200.models.kimi_linear import random_kda_state
    from eredu_b200.models.deepseek import random_mla_state
    from eredu_b200.models.llama import build_from_tensors, build_random
    from eredu_b200.models.moe import make_moe_factory

    if cfg.model_type != "kimi_linear":
        return build_random(cfg, DEV, BF, seed=0)
    out: dict = {}

    def mat(name, *shape):
        out[name] = torch.randn(*shape, device=DEV, dtype=BF) * 0.02

    def ones(name, n):
        out[name] = torch.ones(n)

    mat("model.embed_tokens.weight", cfg.vocab_size, cfg.hidden_size)
    mat("lm_head.weight", cfg.vocab_size, cfg.hidden_size)
    ones("model.norm.weight", cfg.hidden_size)
    made: set = set()

    def layer(li):                                             # one layer's tensors at a time
        p = f"model.layers.{li}."
        for k in [k for k in out if k.startswith("model.layers.")]:
            del out[k]
        ones(p + "input_layernorm.weight", cfg.hidden_size)
        ones(p + "post_attention_layernorm.weight", cfg.hidden_size)
        if cfg.layer_is_kda(li):
            random_kda_state(cfg, p, mat, ones, out, 0.02)
        else:
            random_mla_state(cfg, p, mat, ones)
        mat(p + "mlp.gate.weight", cfg.num_experts, cfg.hidden_size)
        mat(p + "mlp.experts.gate_up_proj", cfg.num_experts, 2 * cfg.moe_intermediate_size, cfg.hidden_size)
        mat(p + "mlp.experts.down_proj", cfg.num_experts, cfg.hidden_size, cfg.moe_intermediate_size)

    def need(name):
        if name.startswith("model.layers."):
            li = int(name.split(".")[2])
            if li not in made:
                made.add(li)
                layer(li)

    def get(name):
        need(name)
        return out[name]

    def has(name):
        need(name)
        return name in out

    return build_from_tensors(cfg, get, has, DEV, BF, moe_factory=make_moe_factory())


# ---------------------------------------------------------------------------------------------- kernels
def kernel_numbers(size: str, T: int = 8192, Bn: int = 32, context: int = 2048, only: str = "") -> list:
    W, _, H, D, P, V, R, Q, RH, dk, dv, E, top, G, keep, ff = SIZES[size]
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

    ones, zeros = torch.ones(W, device=DEV), torch.zeros(W, device=DEV)
    inv = torch.rand(P // 2, device=DEV)
    for phase, M in (("prefill", T), ("decode", Bn)):
        prefill = phase == "prefill"
        ids = torch.stack([torch.randperm(E, device=DEV)[:top] for _ in range(M)]).int() if M <= 64 else \
            torch.rand(M, E, device=DEV).topk(top, -1).indices.int()
        wts = torch.rand(M, top, device=DEV)
        plan = moe_ops.ExpertPlan(ids, top, 0, E, 16, M * top)

        # ---- stream + experts + norm, beside the two kernels that do the same with a bf16 stream
        def norm(i):
            x, y, r = rnd(M, W, dt=F32), rnd(M, W), rnd(M * top, W)
            routed = moe_ops.RoutedRows(r, plan.route_pos, wts)
            return lambda: ops.residual_norm(x, y, routed, ones, zeros, 1e-5, BF)

        def like_norm(i):
            x, y, r, o = rnd(M, W), rnd(M, W), rnd(M * top, W), torch.empty(M, W, device=DEV, dtype=BF)

            def run():
                native.lib().eredu_moe_combine(*map(native.ptr, (r, plan.route_pos, wts, x, None, o)), M, top, W, native.stream_ptr(DEV))
                ops.rmsnorm(y, ones, 1e-5, residual=o)
            return run

        add(f"{phase} residual_norm (stream + mixer + {top} expert rows, LayerNorm)", M * W * (12 + 2 * top), 0, norm, "moe_combine, then rmsnorm + residual", like_norm,
            M * W * (2 * top + 12))

        # ---- routing by groups
        def route(i, groups=(G, keep)):
            z = rnd(M, E + 2 * RH, dt=F32)
            if prefill:
                return lambda: moe_ops.route(z[:, 2 * RH:], top, "sigmoid", False, 1.0, None, *groups)
            x = rnd(M, W)
            return lambda: moe_ops.route_plan_gather(z[:, 2 * RH:], x, top, "sigmoid", False, 1.0, None, 0, E, *groups)

        nb = M * (E * 4 + top * 8) if prefill else M * (E * 4 + W * 2 + top * (8 + 2 * W))
        add(f"{phase} routing by groups" + ("" if prefill else ", plan and gather"), nb, 0, route, "the same without groups", lambda i: route(i, (1, 1)))

        # ---- latents of queries, keys and values
        ctx = T if prefill else context
        bt = batch_of(T, 1, T, True) if prefill else batch_of(1, Bn, context, False)
        pages = int(bt.block_table.max()) + 1
        pool = lambda: rnd(pages, 1, 16, R + P)                                                  # noqa: E731
        qn, kn = torch.ones(Q, device=DEV), torch.ones(R, device=DEV)
        NP = H * V + Q + R + P

        def prep(i):
            x, c = rnd(M, NP), pool()
            return lambda: ops.latent_prepare(x[:, H * V:], Q, R, P, qn, kn, 1e-5, bt.positions, bt.slots, inv, c)

        hq, hk, hd = 16, 4, 128
        hw, gw, hinv = torch.ones(hq * hd, device=DEV), torch.ones(hk * hd, device=DEV), torch.rand(hd // 2, device=DEV)

        def like_prep(i):
            x, kc, vc = rnd(M, (hq + 2 * hk) * hd), rnd(pages, hk, 16, hd), rnd(pages, hk, 16, hd)
            return lambda: ops.qkv_prepare(x, bt.positions, bt.slots, hinv, kc, vc, hq, hk, hd, hd, hw, gw, 1e-5)

        add(f"{phase} latent_prepare", M * (Q + R + P) * 4, 0, prep, "qkv_prepare (norms over whole projections)", like_prep, M * (hq + 2 * hk) * hd * 4)

        uk, uv, up = rnd(H, R, D, s=0.05), rnd(H, V, R, s=0.05), rnd(H * (D + V), R, s=0.05)
        sinks = torch.zeros(H, device=DEV)
        if prefill:
            def turn(i):
                q = rnd(M, H * (D + P))
                return lambda: native.lib().eredu_rotate_heads(q.data_ptr(), bt.positions.data_ptr(), inv.data_ptr(), M, q.stride(0), H, D + P, D, P,
                                                               native.stream_ptr(DEV))

            add("prefill rotate_heads", M * H * P * 4, 0, turn)
            slots = bt.slots

            def gather(i):
                c, o = pool(), torch.empty(T, R + P, device=DEV, dtype=BF)
                return lambda: native.lib().eredu_gather_rows(c.data_ptr(), slots.data_ptr(), o.data_ptr(), T, R + P, 2, native.stream_ptr(DEV))

            add("prefill gather_rows", T * (R + P) * 4, 0, gather)
            # ---- attention over expanded keys and values
            pairs = WINDOW * T - WINDOW * WINDOW / 2
            table = torch.tensor([[0, T, 0, T]], dtype=torch.int32, device=DEV)

            def attn(i):
                q, kv, c, g, o = rnd(T, H * (D + P)), rnd(T, H * (D + V)), rnd(T, R + P), rnd(T, NP), torch.empty(T, H, V, device=DEV, dtype=BF)
                return lambda: native.lib().eredu_attn_prefill_rows(
                    q.data_ptr(), kv.data_ptr(), kv.data_ptr() + H * D * 2, c.data_ptr() + R * 2, g.data_ptr(), sinks.data_ptr(), o.data_ptr(),
                    table.data_ptr(), 1, T, T, T, H, D, P, V, WINDOW, H * (D + P), H * (D + V), R + P, NP, (D + P) ** -0.5,
                    native.status_word(DEV).data_ptr(), native.stream_ptr(DEV))

            lk = 128 if D + P > 64 else 64

            def like_attn(i):
                q, kc, vc = rnd(T, H, lk), rnd(pages, H, 16, lk), rnd(pages, H, 16, lk)
                return lambda: ops.attention_prefill(q, kc, vc, bt.block_table, bt.seq_lens, bt.cu_q, T, lk ** -0.5, window=WINDOW)

            add("prefill latent attention, expanded", T * H * (D + P + D + 3 * V) * 2 + T * P * 2, 2 * pairs * H * (D + P + V), attn,
                f"attention, head size {lk}, same window", like_attn, T * H * 4 * lk * 2, 4 * pairs * H * lk)
        else:
            seen = min(WINDOW, context)

            def attn(i):
                qa, c, o = rnd(Bn, H, R + P), pool(), torch.empty(Bn, H, R, device=DEV, dtype=BF)
                tile, per_sm = latent_ops.latent_tile(H, R, P)
                sp = latent_ops.latent_splits(Bn, -(-H // tile), seen, per_sm * 148)
                return lambda: native.lib().eredu_latent_attn(qa.data_ptr(), c.data_ptr(), o.data_ptr(), bt.block_table.data_ptr(), bt.seq_lens.data_ptr(),
                                                              None, sinks.data_ptr(), Bn, 1, 1, bt.block_table.stride(0), H, R, P, tile, sp, WINDOW,
                                                              (D + P) ** -0.5, native.status_word(DEV).data_ptr(), native.stream_ptr(DEV))

            def like_attn(i):
                q, kc, vc = rnd(Bn, 4 * hk, hd), rnd(pages, hk, 16, hd), rnd(pages, hk, 16, hd)
                sp = ops.decode_splits(Bn, hk, WINDOW)
                return lambda: ops.attention_decode(q, kc, vc, bt.block_table, bt.seq_lens, 1, 0.1, splits=sp, window=WINDOW)

            add("decode latent attention, absorbed", Bn * seen * (R + P) * 2, 2 * Bn * H * seen * (2 * R + P), attn,
                "attention_decode, 4 kv heads of 128, same window", like_attn, Bn * seen * hk * hd * 4, 4 * Bn * seen * 16 * hd)

            # ---- per-head matrices
            def absorb(i):
                q, w, o = rnd(Bn, H, D + P), rnd(H, R, D, s=0.05), torch.empty(Bn, H, R + P, device=DEV, dtype=BF)
                return lambda: ops.head_linear(q, w, o, rot=P, positions=bt.positions, inv_freq=inv)

            def values(i):
                x, w, o, g = rnd(Bn, H, R), rnd(H, V, R, s=0.05), torch.empty(Bn, H, V, device=DEV, dtype=BF), rnd(Bn, NP)
                return lambda: ops.head_linear(x, w, o, gate=g[:, :H * V])

            def like_linear(n, k):
                def make(i):
                    x, w = rnd(Bn, k), rnd(n, k)
                    return lambda: ops.linear(x, w)
                return make

            add("decode head_linear, queries into the latent", H * R * D * 2 + Bn * H * (D + R + 2 * P) * 2, 2 * Bn * H * R * D, absorb, "linear of the same bytes",
                like_linear(H * R, D), H * R * D * 2 + Bn * (D + H * R) * 2)
            add("decode head_linear, latents to gated values", H * V * R * 2 + Bn * H * (R + 2 * V) * 2, 2 * Bn * H * R * V, values, "linear of the same bytes",
                like_linear(V, H * R), H * V * R * 2 + Bn * (V + H * R) * 2)

        # ---- experts
        xs = rnd(M, W)
        gu, dn = rnd(E, 2 * ff, W, s=0.02), rnd(E, W, ff, s=0.02)
        touched = E * (1 - (1 - top / E) ** M)

        def experts(i):
            w1, w2 = (gu, dn) if prefill else (rnd(E, 2 * ff, W, s=0.02), rnd(E, W, ff, s=0.02))
            return lambda: moe_ops.expert_rows(xs, ids, w1, w2)

        add(f"{phase} experts (plan, gather, gate_up + SwiGLU, down)", touched * 3 * W * ff * 2 + M * W * 2 * (1 + 3 * top), 6 * M * top * W * ff, experts)

        # ---- recurrence, beside the gated linear attention and the closest model's scan
        n = 1 if prefill else Bn
        bt = batch_of(M // n, n, M // n, prefill)
        p2s = torch.zeros(int(bt.block_table.max()) + 1, dtype=torch.int32, device=DEV)
        p2s[bt.block_table[:, 0].long()] = torch.arange(n, device=DEV, dtype=torch.int32)
        qk, vw = RH * dk, RH * dv
        size_f = -(-RH * (dk * dv + dk + 1) // 4) * 4
        nw = torch.ones(vw, device=DEV)

        def memory(i):
            x, z, s = rnd(M, 2 * qk + 2 * vw), rnd(M, 2 * RH, dt=F32) + 2.0, torch.zeros(n, size_f, device=DEV)
            return lambda: ops.mlstm(x, z, nw, s, RH, dk, dv, 15.0, 1e-5, bt, p2s)

        gdk, gdv = 128, 128
        GH = RH * dk * dv // (gdk * gdv)
        a2, a2b, gnw = rnd(GH * gdk, 16, dt=F32, s=0.1), rnd(GH * gdk, dt=F32), torch.ones(gdv, device=DEV)

        def gla(i):
            x, s = rnd(M, 2 * GH * (gdk + gdv) + 16), torch.zeros(n, GH, gdk, gdv, device=DEV)
            return lambda: ops.gla_attention(x, a2, a2b, gnw, s, GH, gdk, gdv, 16.0, 1e-5, bt, p2s)

        def delta(i):
            q, k, v = rnd(n, M // n, GH, gdk, s=0.3), rnd(n, M // n, GH, gdk, s=0.1), rnd(n, M // n, GH, gdv)
            ld, be = -torch.rand(n, M // n, GH, gdk, device=DEV) * 0.1, torch.rand(n, M // n, GH, device=DEV)
            s, o = torch.zeros(n, GH, gdk, gdv, device=DEV), torch.empty(n, M // n, GH, gdv, device=DEV, dtype=BF)
            return lambda: native.lib().eredu_gated_delta_scan(*map(native.ptr, (q, k, v, ld, be, s, o)), n, M // n, GH, gdk, gdv, 1, native.stream_ptr(DEV))

        state = n * RH * dk * dv * 8
        io, fl = M * ((2 * qk + 3 * vw) * 2 + RH * 8) + state, 4.0 * M * RH * dk * dv
        gio = M * (2 * GH * gdk + 3 * GH * gdv + 16) * 2 + state
        add(f"{phase} mlstm (gates, recurrence, norm, output gate)", io, fl, memory, "gla_attention, equal state", gla, gio, fl)
        add(f"{phase} mlstm (gates, recurrence, norm, output gate)", io, fl, memory, "gated_delta_scan, vector decay (closest model)", delta,
            M * GH * (2 * gdk + 2 * gdv) * 2 + M * GH * (gdk + 1) * 4 + state, fl)
    native.check_status(DEV)
    return rows


def run(sizes, steps: int, models: bool = True, kernels: bool = True, closest: bool = True) -> dict:
    torch.cuda.set_device(DEV)
    result = {"models": {}, "kernels": {}}
    for size in sizes:
        if models:
            entry = {"lenitar": B.model_numbers(lenitar_config(size), steps, build=random_model)}
            if closest:
                entry["kimi_linear"] = B.model_numbers(closest_config(size), min(steps, 8), build=random_model)
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
