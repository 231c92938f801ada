"""Kasuvik: a decoder with an RMSNorm before and behind every sublayer whose layers mix either by the generalised delta rule or by
attention and a selective scan side by side: ``x <- x + norm1b(mixer(norm1(x)))``, then ``x <- x + norm2b(ff(norm2(x)))``.

The stream is fp32. One kernel (:func:`ops.branch_norm`) normalises what a sublayer returns, adds it and normalises the sum for the
next one, so a sublayer starts from the activations its predecessor left in ``batch.stream``. Projections of one input are fused at
load:

* parallel: ``[q | k | v | x | z]`` -> convolutions, rotation, the append of keys and values (:func:`ops.conv_project`) -> attention
  over a sliding window and the means of the blocks behind it (:func:`ops.pooled_attention`) -> output projection; beside it step
  size, B and C of the convolved x -> :func:`ops.selective_scan` -> output projection. Both outputs are RMS-normed and averaged by
  the kernel that follows.
* general_delta: ``[r | k | v | output gate | removal rate | decay input]`` -> :func:`ops.general_delta` -> output projection.

The feed-forward is gated by a ReLU, which the epilogue of its first GEMM applies. Runs in bf16 and, everything in true 32-bit, in
fp32.
"""
from __future__ import annotations

import math

import torch

from .. import ops
from .rope import base_inv_freq

TOP_LEVEL = {"model.embed_tokens.weight": "embed", "model.norm.weight": "final.norm", "lm_head.weight": "head"}
DEFAULT_DECAY_RANK = 16              # rank of the decay projection in randomly initialised models (checkpoints: the tensor's own)
LOG_DECAY = math.exp(-0.5)           # the strongest decay of a step, as -log


# ---------------------------------------------------------------------------------------------- configuration
def _attention_spec(i: int, m: dict):
    from .config import MixerSpec

    mask, rot = m.get("mask") or {}, m.get("rot") or {}
    s = MixerSpec("attention", heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                  scale=float(m["scale"]), conv=int(m["conv"]), window=int(mask["size"]), pool=int(mask["pool"]),
                  rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 10000.0)))
    if s.kv_heads < 1 or s.heads % s.kv_heads or s.rot_dims % 2 or s.rot_dims > s.dim or s.window < 1 or s.pool < 1 or s.conv < 1:
        raise ValueError(f"Kasuvik layer {i}: inconsistent attention geometry")
    return s


def config_from_dict(cls, d: dict):
    """``config.json`` -> ModelConfig: the layer list becomes ``mixers``, the generic fields describe the whole."""
    from .config import MixerSpec

    mixers = []
    for i, layer in enumerate(d["layers"]):
        kind, m, mlp = layer["type"], layer["mixer"], layer.get("mlp")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"Kasuvik layer {i}: unknown feed-forward {mlp.get('kind')!r}")
        if kind == "general_delta":
            s = MixerSpec(kind, heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["dim"]))
        elif kind == "parallel":
            r = m["right"]
            right = MixerSpec("mamba", width=int(r["inner"]), state=int(r["state"]), dt_rank=int(r["dt_rank"]), conv=int(r["conv"]))
            if min(right.width, right.state, right.dt_rank, right.conv) < 1:
                raise ValueError(f"Kasuvik layer {i}: inconsistent scan geometry")
            s = MixerSpec(kind, left=_attention_spec(i, m["left"]), right=right)
        else:
            raise ValueError(f"Kasuvik layer {i}: unknown mixer {kind!r}")
        s.ff = int(mlp["ff"]) if mlp is not None else 0
        mixers.append(s)
    attn = [s.left for s in mixers if s.kind == "parallel"] or [MixerSpec("attention", 1, 1, 64, 64)]
    return cls(model_type="kasuvik", vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), intermediate_size=max(s.ff for s in mixers),
               num_hidden_layers=len(mixers), num_attention_heads=attn[0].heads, num_key_value_heads=attn[0].kv_heads,
               head_dim=attn[0].dim, rms_norm_eps=float(d["norm"]["eps"]), rope_theta=attn[0].rot_base,
               max_position_embeddings=int(d.get("max_position_embeddings", 1 << 20)), tie_word_embeddings=False,
               embedding_scale=float(d["embedding"]["scale"]), layer_types=[s.kind for s in mixers], eos_token_id=d.get("eos_token_id"),
               bos_token_id=d.get("bos_token_id"), torch_dtype=str(d.get("torch_dtype", "bfloat16")), mixers=mixers)


def config_dict(cfg) -> dict:
    """ModelConfig -> ``config.json`` (inverse of :func:`config_from_dict`)."""
    layers = []
    for s in cfg.mixers:
        if s.kind == "general_delta":
            m = {"heads": s.heads, "dim": s.dim}
        else:
            a, b = s.left, s.right
            m = {"left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "conv": a.conv, "scale": a.scale,
                          "mask": {"size": a.window, "pool": a.pool}, "rot": {"dims": a.rot_dims, "base": a.rot_base}},
                 "right": {"inner": b.width, "state": b.state, "dt_rank": b.dt_rank, "conv": b.conv}}
        layers.append({"type": s.kind, "mixer": m, "mlp": {"kind": "dense", "ff": s.ff} if s.ff else None})
    d = {"architecture": "Kasuvik", "vocab": cfg.vocab_size, "width": cfg.hidden_size, "norm": {"eps": cfg.rms_norm_eps},
         "embedding": {"scale": cfg.embedding_scale}, "layers": layers}
    for k in ("eos_token_id", "bos_token_id"):
        if getattr(cfg, k) is not None:
            d[k] = getattr(cfg, k)
    return d


# ---------------------------------------------------------------------------------------------- tensors
def canonical_access(get, has):
    """The three tensors outside the layers under the names the generic loader asks for."""
    def resolve(name):
        alt = TOP_LEVEL.get(name)
        return alt if alt is not None and has(alt) else name

    return (lambda name: get(resolve(name))), (lambda name: has(resolve(name)))


def tensor_shapes(cfg, decay_rank: int = DEFAULT_DECAY_RANK) -> dict:
    """Every tensor of a checkpoint of this geometry: name -> shape."""
    W = cfg.hidden_size
    out = {"embed": (cfg.vocab_size, W), "head": (cfg.vocab_size, W), "final.norm": (W,)}
    for i, s in enumerate(cfg.mixers):
        p = f"l{i}.mix."
        out.update({f"l{i}.norm1": (W,), f"l{i}.norm1b": (W,)})
        if s.kind == "general_delta":
            n = s.heads * s.dim
            out.update({p + t: (n, W) for t in "rkvga"})
            out.update({p + "a.b": (n,), p + "w1": (decay_rank, W), p + "w2": (n, decay_rank), p + "w0": (n,), p + "norm": (n,), p + "o": (W, n)})
        else:
            a, b, l, r = s.left, s.right, p + "left.", p + "right."
            for t, n in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
                out.update({l + t: (n, W), l + t + ".b": (n,), l + t + ".conv": (n, a.conv)})
            out.update({l + "temp": (a.heads,), l + "o": (W, a.heads * a.vdim), l + "out": (W,)})
            out.update({r + "in": (2 * b.width, W), r + "conv": (b.width, b.conv), r + "conv.b": (b.width,),
                        r + "x": (b.dt_rank + 2 * b.state, b.width), r + "dt": (b.width, b.dt_rank), r + "dt.b": (b.width,),
                        r + "A_log": (b.width, b.state), r + "D": (b.width,), r + "o": (W, b.width), r + "out": (W,)})
        if s.ff:
            q = f"l{i}.mlp."
            out.update({f"l{i}.norm2": (W,), f"l{i}.norm2b": (W,), q + "gate": (s.ff, W), q + "up": (s.ff, W), q + "down": (W, s.ff)})
    return out


def random_tensor(name: str, shape: tuple, generator, std: float = 0.02, device="cpu") -> torch.Tensor:
    """Seeded fp32 values of one tensor: unit norms, temperatures and skips, small step sizes, state decays spread over the states,
    convolutions that keep their input's size, N(0, std) otherwise."""
    last = name.rsplit(".", 1)[-1]
    if "norm" in last or last in ("temp", "D", "out"):
        return torch.ones(shape, dtype=torch.float32, device=device)
    if last == "A_log":
        return torch.log(torch.arange(1, shape[1] + 1, dtype=torch.float32, device=device)).expand(shape).contiguous()
    t = torch.randn(shape, generator=generator, dtype=torch.float32, device=device)
    if last == "conv":
        return t * shape[1] ** -0.5
    return t * std - 4.0 if name.endswith("dt.b") else t * std


def build(model, cfg, get, has, up) -> None:
    """Fill ``model.layers`` (called by the generic loader after the embedding, final norm and head)."""
    from .llama import LayerWeights

    f32 = lambda n: up(get(n), torch.float32)                                          # noqa: E731
    grown = lambda t, rows=0, cols=0: torch.nn.functional.pad(t, (0, cols, 0, rows))   # noqa: E731

    for li, s in enumerate(cfg.mixers):
        p = f"l{li}.mix."
        lw = LayerWeights(attn_norm=f32(f"l{li}.norm1"), wqkv=None, wo=None, ffn_norm=None)
        lw.block_kind = "kasuvik"
        e = lw.extra = {"norm1b": f32(f"l{li}.norm1b")}
        # widths that are no whole number of 16-byte pieces are filled up with zero rows or columns
        if s.kind == "general_delta":
            w1 = get(p + "w1")
            pad = -w1.shape[0] % 8
            mats = [get(p + n) for n in "rkvga"]
            rows = sum(m.shape[0] for m in mats) + w1.shape[0] + pad
            lw.wqkv = up(torch.cat([*mats, grown(w1, pad + -rows % 8)]))
            lw.wo = up(get(p + "o"))
            e.update(w2=up(grown(get(p + "w2"), 0, pad), torch.float32), w0=f32(p + "w0"), rate_b=f32(p + "a.b"), norm=f32(p + "norm"))
        else:
            _build_parallel(model, lw, s, p, get, has, up, grown)
        if s.ff:
            pad = -s.ff % 8
            q = f"l{li}.mlp."
            lw.ffn_norm, e["norm2b"] = f32(f"l{li}.norm2"), f32(f"l{li}.norm2b")
            lw.w_gate_up = up(torch.cat([grown(get(q + n), pad) for n in ("gate", "up")]))
            lw.w_down = up(grown(get(q + "down"), 0, pad))
        model.layers.append(lw)


def _build_parallel(model, lw, s, p, get, has, up, grown) -> None:
    a, b, e = s.left, s.right, lw.extra
    f32 = lambda n: up(get(n), torch.float32)                                          # noqa: E731
    l, r = p + "left.", p + "right."
    mats = [get(l + n) for n in "qkv"] + [get(r + "in")]
    biases = [get(l + n + ".b") if has(l + n + ".b") else torch.zeros_like(m[:, 0]) for n, m in zip("qkv", mats)]
    pad = -sum(m.shape[0] for m in mats) % 8
    mats[-1] = grown(mats[-1], pad)
    lw.wqkv = up(torch.cat(mats))
    lw.bqkv = up(torch.cat([*biases, torch.zeros_like(mats[-1][:, 0])]))
    lw.wo = up(get(l + "o"))
    taps = up(torch.cat([get(l + n + ".conv") for n in "qkv"]).t(), torch.float32)
    temp = f32(l + "temp") if has(l + "temp") else None
    inv = base_inv_freq(a.rot_base, a.rot_dims) if a.rot_dims else torch.zeros(0)
    scan = b.state_shape[0]
    e["heads"] = dict(taps=taps, n_q=a.heads, n_kv=a.kv_heads, dk=a.dim, dv=a.vdim, q_scale=temp, pool=a.pool, hist=scan,
                      inv_freq=inv.to(device=model.device, dtype=torch.float32))
    e["channels"] = ops.ConvChannels(up(get(r + "conv").t(), torch.float32), f32(r + "conv.b") if has(r + "conv.b") else None,
                                     a.conv_channels, hist=scan - b.conv_elems)
    # [step size input | B | C], the step size's part filled up so that it is the input of a GEMM as it lies
    x, dt = get(r + "x"), get(r + "dt")
    rank, fill = b.dt_rank, -b.dt_rank % 8
    x = torch.cat((grown(x[:rank], fill), x[rank:]))
    e.update(x=up(grown(x, -x.shape[0] % 8)), dt=up(grown(dt, 0, fill)), dt_b=f32(r + "dt.b"), A=-torch.exp(f32(r + "A_log")), D=f32(r + "D"),
             right_o=up(get(r + "o")), out=(f32(l + "out"), f32(r + "out")))


# ---------------------------------------------------------------------------------------------- forward
def enter(model, batch):
    """The scaled embedding as the start of the fp32 stream, and the first layer's input."""
    x = ops.embedding_stream(batch.token_ids, model.embed, scale=model.cfg.embedding_scale, want_act=False)[0]
    batch.stream = (x, _normed(model, model.layers[0].attn_norm, x))
    return x


def _normed(model, weight, x):
    return ops.residual_norm(x, weight=weight, eps=model.cfg.rms_norm_eps, act_dtype=model.dtype, center=False)[1]


def block_forward(model, li, lw, x, batch, kv):
    s, i, eps = model.cfg.mixers[li], li - model.first_layer, model.cfg.rms_norm_eps
    # the activations the previous layer left, unless somebody replaced the stream
    h = batch.stream[1] if batch.stream is not None and batch.stream[0] is x else _normed(model, lw.attn_norm, x)
    following = model.layers[i + 1].attn_norm if i + 1 < len(model.layers) else None
    after = lw.ffn_norm if s.ff else following
    if s.kind == "general_delta":
        x, h = ops.branch_norm(x, [_general_delta(model, li, lw, s, h, batch, kv)], lw.extra["norm1b"], after, eps, model.dtype)
    else:
        x, h = ops.branch_norm(x, _parallel(model, li, lw, s, h, batch, kv), lw.extra["norm1b"], after, eps, model.dtype,
                               branch_weights=lw.extra["out"], gain=0.5)
    if s.ff:
        y = ops.linear(ops.gated_linear(h, lw.w_gate_up, lw.w_gate_up.shape[0] // 2, activation="relu"), lw.w_down)
        x, h = ops.branch_norm(x, [y], lw.extra["norm2b"], following, eps, model.dtype)
    batch.stream = (x, h) if following is not None else None
    return x


def final_norm(model, x):
    """The normalised rows the output head reads."""
    return _normed(model, model.final_norm, x)


def _parallel(model, li, lw, s, h, batch, kv):
    a, b, e = s.left, s.right, lw.extra
    proj = ops.linear(h, lw.wqkv, bias=lw.bqkv)
    k_cache, v_cache = kv.layer(li)
    pooled, state = kv.pooled[li], kv.layer_state[li]
    c = e["channels"]
    q, x = ops.conv_project(proj, state, batch, kv.page_to_slot, ops.ConvHeads(**e["heads"], k_cache=k_cache, v_cache=v_cache, pooled=pooled), c)
    attn = ops.pooled_attention(q, k_cache, v_cache, pooled, batch, a.scale, a.window, a.pool)
    left = ops.linear(attn.view(attn.shape[0], -1), lw.wo)
    y = ops.selective_scan(x, proj[:, c.start + b.width:c.start + 2 * b.width], ops.linear(x, e["x"]), e["dt"].shape[1], e["dt"], e["dt_b"],
                           e["A"], e["D"], state, batch, kv.page_to_slot)
    return [left, ops.linear(y, e["right_o"])]


def _general_delta(model, li, lw, s, h, batch, kv):
    e = lw.extra
    y = ops.general_delta(ops.linear(h, lw.wqkv), e["w2"], e["w0"], e["rate_b"], e["norm"], kv.layer_state[li], s.heads, s.dim, s.vdim, LOG_DECAY,
                          model.cfg.rms_norm_eps, batch, kv.page_to_slot)
    return ops.linear(y, lw.wo)
