"""Nidozen at sizes that resemble a real model's layers, beside the framework's closest model at equal size (Nemotron-H: the
same widths, attention geometry, recurrent-state size and squared-ReLU feed-forwards), and its kernels beside the like
kernels of that and the other families, each against its roofline.

    python -m benchmarks.bench_nidozen [--sizes small medium large] [--no-kernels] [--no-models]
    python bench.py --design nidozen

Random weights, bf16. Models: prefill of one prompt (CUDA events around ``Engine.prefill``), decode steps as captured CUDA
graphs (events around ``--steps`` replays after warm-up); every model's weights exceed L2. Kernels: a captured graph of launches
over separate buffers that together exceed L2, so that nothing is found in the cache; time per launch.
"""
from __future__ import annotations

import argparse
import json
from pathlib import Path

import torch

from eredu_b200 import ops
from eredu_b200.models.config import ModelConfig
from eredu_b200.models.llama import ForwardBatch, build_from_tensors, build_random
from eredu_b200.models.nemotron_h import random_block_state
from eredu_b200.ops import SamplingParams, native
from eredu_b200.runtime.engine import Engine

DEV = torch.device("cuda:0")
BF, F32 = torch.bfloat16, torch.float32
# width, groups of four layers, query heads, kv heads, head size, recurrent heads, state rows (keys), state columns (values)
SIZES = {"small": (1024, 4, 16, 4, 64, 8, 64, 128), "medium": (2048, 4, 16, 4, 128, 16, 128, 128), "large": (4096, 4, 32, 8, 128, 32, 128, 128)}
CHUNK = 1024
VOCAB = 32000


def nidozen_config(size: str) -> ModelConfig:
    W, n, H, G, D, R, dk, dv = SIZES[size]
    mlp = {"kind": "dense", "ff": 3 * W}
    at = {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "mask": {"size": CHUNK}, "rot": {"dims": D // 2, "base": 10000.0}, "scale": D ** -0.5}
    layers = []
    for i in range(n):
        layers += [{"type": "mingru", "mixer": {"width": R * dv}, "mlp": mlp}, {"type": "attention", "mixer": at, "mlp": mlp},
                   {"type": "attention", "mixer": {**at, "kv_from": 4 * i + 1}, "mlp": mlp},
                   {"type": "gla", "mixer": {"heads": R, "dim": dk, "vdim": dv, "tau": 16.0}, "mlp": mlp}]
    return ModelConfig.from_hf_dict({"architecture": "Nidozen", "width": W, "vocab": VOCAB, "norm": {"eps": 1e-5}, "layers": layers})


def closest_config(size: str) -> ModelConfig:
    W, n, H, G, D, R, dk, dv = SIZES[size]
    return ModelConfig.from_hf_dict({
        "model_type": "nemotron_h", "hybrid_override_pattern": "M-*-*-M-" * n, "hidden_size": W, "num_attention_heads": H,
        "num_key_value_heads": G, "head_dim": D, "mamba_num_heads": R, "mamba_head_dim": dv, "ssm_state_size": dk, "n_groups": min(8, R),
        "conv_kernel": 4, "intermediate_size": 3 * W, "vocab_size": VOCAB, "n_routed_experts": 0, "layer_norm_epsilon": 1e-5,
        "max_position_embeddings": 65536})


def random_model(cfg: ModelConfig):
    """Random weights drawn on the device."""
    if cfg.model_type != "nemotron_h":
        return build_random(cfg, DEV, BF, seed=0)
    out: dict = {}

    def mat(name, *shape):
        out[name] = torch.randn(*shape, device=DEV, dtype=BF) * 0.02

    mat("model.embed_tokens.weight", cfg.vocab_size, cfg.hidden_size)
    mat("lm_head.weight", cfg.vocab_size, cfg.hidden_size)
    out["model.norm.weight"] = torch.ones(cfg.hidden_size)
    for li in range(cfg.num_hidden_layers):
        random_block_state(cfg, li, f"model.layers.{li}.", mat, out, 0.02)
    return build_from_tensors(cfg, out.__getitem__, out.__contains__, DEV, BF)


def timed(fn, reps: int) -> float:
    """Milliseconds per call."""
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(reps):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / reps


def model_numbers(cfg: ModelConfig, steps: int, prefills=(2048, 8192), batches=(1, 32), context: int = 2048, build=random_model) -> dict:
    model = build(cfg)
    eng = Engine(model, max_batch=max(batches), max_seq_len=max(max(prefills), context + steps + 64) + 16,
                 num_pages=max(batches) * ((context + steps + 64) // 16 + 2) + max(prefills) // 16 + 8, prefill_chunk=16384)
    g = torch.Generator().manual_seed(0)
    greedy = SamplingParams(temperature=0.0)
    out = {"weight_gb": round(model.weight_bytes() / 1e9, 2), "prefill_tokens_per_s": {}, "decode_tokens_per_s": {}, "launches_per_step": None}
    for T in prefills:
        p = torch.randint(0, VOCAB, (T,), generator=g).tolist()
        times = []
        for i in range(5):
            s = eng.new_sequence(p, greedy, max_new_tokens=1)
            ms = timed(lambda: eng.prefill([s]), 1)
            eng.release(s)
            if i >= 2:
                times.append(ms)
        out["prefill_tokens_per_s"][T] = round(T / sorted(times)[1] * 1e3)
    for B in batches:
        seqs = [eng.new_sequence(torch.randint(0, VOCAB, (context,), generator=g).tolist(), greedy, max_new_tokens=steps + 32) for _ in range(B)]
        eng.start_decode(seqs, eng.prefill(seqs))
        for _ in range(8):
            eng.decode_step(sync=False)
        ms = timed(lambda: eng.decode_step(sync=False), steps)
        out["decode_tokens_per_s"][B] = round(B / ms * 1e3)
        if out["launches_per_step"] is None:
            n0, graph = native.launch_count(), eng.use_graph
            eng.use_graph = False
            eng.decode_step(sync=False)
            eng.use_graph = graph
            out["launches_per_step"] = native.launch_count() - n0
        for s in seqs:
            eng.release(s)
        eng._decode_state = None
    native.check_status(DEV)
    del eng, model
    torch.cuda.empty_cache()
    return out


# ---------------------------------------------------------------------------------------------- kernels
def peaks() -> tuple:
    f = Path(__file__).resolve().parent.parent / "MEASURED_PEAKS.json"
    d = json.loads(f.read_text()) if f.exists() else {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    return d["hbm_gbs"], d["bf16_tflops"]


def per_launch_us(make, nbytes: float, reps: int = 5) -> float:
    """``make(i)`` -> a closure over buffers of its own; enough of them that a pass exceeds L2 three times over."""
    n = max(2, min(48, int(4e8 / max(nbytes, 1)) + 1))
    calls = [make(i) for i in range(n)]
    for c in calls:
        c()
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for c in calls:
            c()
    for _ in range(3):
        graph.replay()
    us = timed(graph.replay, reps) * 1e3 / n
    del graph, calls
    torch.cuda.empty_cache()
    return us


def rnd(*shape, dt=BF, s=1.0):
    return (torch.randn(*shape, device=DEV, dtype=F32) * s).to(dt)


def batch_of(rows: int, batch: int, kv_len: int, prefill: bool) -> ForwardBatch:
    """``batch`` sequences of ``rows`` new tokens each at the end of ``kv_len`` cached ones, pages in order."""
    pages = (kv_len + 15) // 16
    bt = (torch.arange(batch * pages, device=DEV, dtype=torch.int32) + 1).view(batch, pages)
    pos = torch.arange(kv_len - rows, kv_len, device=DEV).repeat(batch)
    slots = torch.cat([bt[b].long()[pos[:rows] // 16] * 16 + pos[:rows] % 16 for b in range(batch)])
    cu = torch.arange(batch + 1, device=DEV, dtype=torch.int32) * rows
    return ForwardBatch(token_ids=None, positions=pos.int(), slots=slots, block_table=bt, seq_lens=torch.full((batch,), kv_len, device=DEV, dtype=torch.int32),
                        is_prefill=prefill, cu_q=cu if prefill else None, max_q_len=rows, q_per_seq=rows, max_kv_len=kv_len, sm_count=148)


def kernel_numbers(size: str, T: int = 8192, B: int = 32, context: int = 2048) -> list:
    W, _, H, G, D, R, dk, dv = SIZES[size]
    bw, tf = peaks()
    rows = []

    def add(name, like, nbytes, flops, make, like_make, like_bytes=None, like_flops=None):
        us = per_launch_us(make, nbytes)
        roof = max(nbytes / bw / 1e3, flops / tf / 1e6)
        entry = {"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "x": round(us / roof, 2)}
        if like_make is not None:
            lb, lf = like_bytes or nbytes, like_flops if like_flops is not None else flops
            lus = per_launch_us(like_make, lb)
            lroof = max(lb / bw / 1e3, lf / tf / 1e6)
            entry.update(like=like, like_us=round(lus, 2), like_roofline_us=round(lroof, 2), like_x=round(lus / lroof, 2),
                         relative=round(us / roof / (lus / lroof), 2))
        rows.append(entry)
        print(json.dumps(entry), flush=True)

    one, vec = torch.ones(1, device=DEV), torch.ones(W, device=DEV)
    inv = torch.rand(D // 4, device=DEV)
    for phase, M in (("prefill", T), ("decode", B)):
        # ---- norm of a sublayer's output + fp32 residual, beside RMSNorm with a bf16 residual
        def norm(i):
            y, x = rnd(M, W), rnd(M, W, dt=F32)
            return lambda: ops.rms_residual(y, one, 1e-5, residual=x, act_dtype=BF)

        def like_norm(i):
            y, x = rnd(M, W), rnd(M, W)
            return lambda: ops.rmsnorm(y, vec, 1e-5, residual=x)

        add(f"{phase} rms_residual", "rmsnorm + residual", M * W * 12, 0, norm, like_norm, M * W * 8)
        # ---- squared-ReLU linear beside the plain one
        wu = rnd(3 * W, W, s=0.02)

        def up(i, act="relu2"):
            x, w = rnd(M, W), wu if phase == "prefill" else rnd(3 * W, W, s=0.02)
            return lambda: ops.linear(x, w, activation=act)

        nb = (M * W * 4 + 3 * W * W) * 2
        add(f"{phase} linear + relu2", "linear", nb, 6 * M * W * W, up, lambda i: up(i, None))
        # ---- query / key / value preparation beside RoPE + append
        Q = H * D + 2 * G * D
        qw, kw = torch.ones(H * D, device=DEV), torch.ones(G * D, device=DEV)
        hw = torch.ones(D, device=DEV)
        kv = batch_of(T, 1, T, True) if phase == "prefill" else batch_of(1, B, context, False)
        n_pages = int(kv.block_table.max()) + 1
        pool = lambda: torch.zeros(n_pages, G, 16, D, device=DEV, dtype=BF)                    # noqa: E731

        def prep(i):
            x, kc, vc = rnd(M, Q), pool(), pool()
            return lambda: ops.qkv_prepare(x, kv.positions, kv.slots, inv, kc, vc, H, G, D, D, qw, kw, 1e-5, value_norm=True)

        def like_prep(i):
            x, kc, vc = rnd(M, Q), pool(), pool()
            return lambda: ops.rope_kv(x, kv.positions, kv.slots, inv, kc, vc, H, G, D, rot=D // 2, q_norm_w=hw, k_norm_w=hw)

        if phase == "prefill":           # decode steps prepare inside the attention kernel
            add(f"{phase} qkv_prepare", "rope_kv (per-head norms)", M * Q * 4, 0, prep, like_prep)
        # ---- attention
        n = T if phase == "prefill" else context
        if phase == "prefill":
            pairs, like_pairs = n // CHUNK * CHUNK * CHUNK / 2, n * n / 2

            def attn(i, chunk=CHUNK):
                q, kc, vc = rnd(T, H, D), rnd(n_pages, G, 16, D), rnd(n_pages, G, 16, D)
                return lambda: ops.attention_prefill(q, kc, vc, kv.block_table, kv.seq_lens, kv.cu_q, T, D ** -0.5, chunk=chunk)

            io = T * (2 * H + 2 * G) * D * 2
            add("prefill attention, chunks", "full causal attention", io, 4 * pairs * H * D, attn, lambda i: attn(i, 0), io, 4 * like_pairs * H * D)
            add("prefill attention, chunks", "sliding window of a chunk", io, 4 * pairs * H * D, attn, window_attention(T, n_pages, H, G, D, kv), io,
                4 * H * D * (CHUNK * n - CHUNK * CHUNK / 2))
        else:
            lo = (context - 1) % CHUNK + 1
            sp = kv.layer_splits(G, CHUNK)

            def attn(i):
                x, kc, vc = rnd(B, Q), rnd(n_pages, G, 16, D), rnd(n_pages, G, 16, D)
                return lambda: ops.attention_decode_rope(x, kc, vc, kv.block_table, kv.seq_lens, 1, D ** -0.5, kv.positions, kv.slots, inv, H, G, D,
                                                         q_norm_w=qw, k_norm_w=kw, norm_eps=1e-5, splits=sp, chunk=CHUNK, value_dim=D,
                                                         norm_whole=True, value_norm=True)

            def like_attn(i, window=0):
                x, kc, vc = rnd(B, Q), rnd(n_pages, G, 16, D), rnd(n_pages, G, 16, D)
                sl = ops.decode_splits(B, G, window or context)
                return lambda: ops.attention_decode_rope(x, kc, vc, kv.block_table, kv.seq_lens, 1, D ** -0.5, kv.positions, kv.slots, inv, H, G, D,
                                                         rot=D // 2, q_norm_w=hw, k_norm_w=hw, norm_eps=1e-5, splits=sl, window=window)

            add("decode attention from the projection, chunks", "the same, full context, per-head norms", B * lo * G * D * 4, 0, attn, like_attn,
                B * context * G * D * 4, 0)
            add("decode attention from the projection, chunks", "the same, window of a chunk, per-head norms", B * lo * G * D * 4, 0, attn,
                lambda i: like_attn(i, CHUNK), B * CHUNK * G * D * 4, 0)
    recurrent_numbers(size, add, T, B)
    return rows


def window_attention(T, n_pages, H, G, D, kv):
    def make(i):
        q, kc, vc = rnd(T, H, D), rnd(n_pages, G, 16, D), rnd(n_pages, G, 16, D)
        return lambda: ops.attention_prefill(q, kc, vc, kv.block_table, kv.seq_lens, kv.cu_q, T, D ** -0.5, window=CHUNK)

    return make


def recurrent_numbers(size, add, T, B) -> None:
    """Recurrences beside the Mamba-2 scan (the operator the closest model runs) and the gated-delta kernel."""
    _, _, _, _, _, R, dk, dv = SIZES[size]
    qk, vw, rank = R * dk, R * dv, 16
    a2, a2_b, nw = rnd(qk, rank, dt=F32, s=0.1), rnd(qk, dt=F32), torch.ones(dv, device=DEV)
    p2s = torch.zeros(B * 8 + 2048, dtype=torch.int32, device=DEV)
    for phase, M, n in (("prefill", T, 1), ("decode", B, B)):
        bt = batch_of(M // n, n, M // n, phase == "prefill")
        p2s[bt.block_table[:, 0].long()] = torch.arange(n, device=DEV, dtype=torch.int32)
        state = n * R * dk * dv * 8

        def gla(i):
            x, s = rnd(M, 2 * qk + 2 * vw + rank), torch.zeros(n, R, dk, dv, device=DEV)
            return lambda: ops.gla_attention(x, a2, a2_b, nw, s, R, dk, dv, 16.0, 1e-5, bt, p2s)

        io = M * (2 * qk + 3 * vw + rank) * 2 + state

        def mamba(i):
            x, b, c = rnd(n, M // n, R, dv), rnd(n, M // n, min(8, R), dk, s=0.3), rnd(n, M // n, min(8, R), dk, s=0.3)
            dt, A, Dv = torch.rand(n, M // n, R, device=DEV) * 0.1, -torch.rand(R, device=DEV), torch.ones(R, device=DEV)
            s, out = torch.zeros(n, R, dv, dk, device=DEV), torch.empty(n, M // n, R, dv, device=DEV, dtype=BF)
            if phase == "prefill":
                return lambda: ops.mamba2_scan(x, b, c, dt, A, Dv, s)
            return lambda: native.lib().eredu_mamba2_scan(*map(native.ptr, (x, b, c, dt, A, Dv, s, out)), n, M // n, R, min(8, R), dv, dk,
                                                          native.stream_ptr(DEV))

        def delta(i):
            q, k, v = rnd(n, M // n, R, dk, s=0.3), rnd(n, M // n, R, dk, s=0.1), rnd(n, M // n, R, dv)
            ld, be = -torch.rand(n, M // n, R, dk, device=DEV) * 0.1, torch.rand(n, M // n, R, device=DEV)
            s, out = torch.zeros(n, R, dk, dv, device=DEV), torch.empty(n, M // n, R, dv, device=DEV, dtype=BF)
            return lambda: native.lib().eredu_gated_delta_scan(*map(native.ptr, (q, k, v, ld, be, s, out)), n, M // n, R, dk, dv, 1,
                                                               native.stream_ptr(DEV))

        mio = M * (2 * vw + 2 * min(8, R) * dk + 2 * R) * 2 + state
        dio = M * (2 * qk + 2 * vw) * 2 + M * (qk + R) * 4 + state
        flops = 4.0 * M * R * dk * dv
        add(f"{phase} gla (decay, recurrence, norm, gate)", "mamba2_scan", io, flops, gla, mamba, mio, flops)
        add(f"{phase} gla (decay, recurrence, norm, gate)", "gated_delta_scan, vector decay", io, flops, gla, delta, dio, flops)

        def mingru(i):
            x, s = rnd(M, 3 * vw), torch.zeros(n, vw, device=DEV)
            return lambda: ops.mingru_scan(x, s, vw, bt, p2s)

        def conv(i):
            x, s = rnd(M, vw), torch.zeros(n, 3, vw, device=DEV, dtype=BF)
            w, slot = torch.ones(vw, 4, device=DEV), torch.arange(n, device=DEV, dtype=torch.int32).view(-1, 1).contiguous()
            return lambda: ops.short_conv(x, w, None, s, slot, bt.cu_q, bt.q_per_seq, bt.positions, bt.slots, M // n, mode=1)

        add(f"{phase} mingru", "mamba2_scan", M * vw * 8 + n * vw * 8, 0, mingru, mamba, mio, flops)
        add(f"{phase} mingru", "short_conv", M * vw * 8 + n * vw * 8, 0, mingru, conv, M * vw * 4 + n * vw * 12, 0)


def run(sizes, steps: int, models: bool = True, kernels: bool = True) -> dict:
    torch.cuda.set_device(DEV)
    result = {"models": {}, "kernels": {}}
    for size in sizes:
        if models:
            ours, other = model_numbers(nidozen_config(size), steps), model_numbers(closest_config(size), steps)
            result["models"][size] = {"nidozen": ours, "nemotron_h": other}
            print(json.dumps({"size": size, **result["models"][size]}), flush=True)
        if kernels:
            result["kernels"][size] = kernel_numbers(size)
    return result


def main() -> None:
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", nargs="*", default=list(SIZES), choices=list(SIZES))
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--no-models", action="store_true")
    ap.add_argument("--no-kernels", action="store_true")
    a = ap.parse_args()
    run(a.sizes, a.steps, not a.no_models, not a.no_kernels)


if __name__ == "__main__":
    main()
