"""Gulazen: a decoder whose sublayers read the residual stream as it is and are normed on their output:
``x <- x + s1 * norm1(mixer(x + conv(x)))``, ``x <- x + s2 * norm2(ff(x))``.

The stream is fp32 and starts from the embedding plus sinusoidal position vectors; nothing else knows positions. A norm's weight (stored
as the distance from one) and the layer scale behind it are one vector after loading, so a single kernel (:func:`ops.rms_residual`)
normalises what a sublayer returns - the weighted rows of routed experts and the shared expert added up on the way -, adds it to the
stream and writes the copy the next projections read. In decode steps it also applies the causal convolution in front of the next
layer's mixer; prompts run it on its own (:func:`ops.stream_conv`). Its last inputs are fp32 state, one slot per sequence.

Attention: ``[q | k | v]`` -> norms over the whole q and the whole k, append (:func:`ops.qkv_prepare`) -> scores of all heads, capped and
mixed across heads before a softmax with sinks over a sliding window and the first tokens (:func:`ops.talking_attention`) -> output
projection. Feed-forward: xIELU in the epilogue of the up projection, or softmax-routed SwiGLU experts beside a shared one.

Runs in bf16 and, everything in true 32-bit, in fp32.
"""
from __future__ import annotations

import torch

from .. import ops
from .rope import base_inv_freq

TOP_LEVEL = {"model.embed_tokens.weight": "embed", "model.norm.weight": "final.norm"}
POSITION_BASE = 10000.0              # wavelengths of the position vectors run from 2 pi towards 2 pi times this


# ---------------------------------------------------------------------------------------------- configuration
def _feed_forward(i: int, mlp):
    """(dense width, routed experts) of a layer."""
    from .config import RoutedSpec

    if mlp is None:
        return 0, None
    if mlp["kind"] == "dense":
        return int(mlp["ff"]), None
    if mlp["kind"] != "moe":
        raise ValueError(f"Gulazen layer {i}: unknown feed-forward {mlp['kind']!r}")
    r = mlp["router"]
    spec = RoutedSpec(int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"]), router_scoring="topk_softmax",
                      shared_ff=int((mlp.get("shared") or {}).get("ff", 0)))
    if not 1 <= spec.num_experts_per_tok <= spec.num_experts:
        raise ValueError(f"Gulazen layer {i}: {spec.num_experts_per_tok} of {spec.num_experts} experts")
    return 0, spec


def config_from_dict(cls, d: dict):
    """``config.json`` -> ModelConfig: the layer list becomes ``mixers``, the generic fields describe the whole."""
    from .config import MixerSpec

    mixers, width, taps = [], int(d["width"]), int((d.get("canon") or {}).get("taps", 0))
    for i, layer in enumerate(d["layers"]):
        m = layer["mixer"]
        if layer["type"] != "attention":
            raise ValueError(f"Gulazen layer {i}: unknown mixer {layer['type']!r}")
        mask = m.get("mask") or {}
        s = MixerSpec("attention", heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                      scale=float(m["scale"]), softcap=float(m.get("softcap") or 0.0), window=int(mask.get("size", 0)),
                      keep_first=int(mask.get("keep_first", 0)), lead_conv=taps, lead_width=width)
        s.ff, s.moe = _feed_forward(i, layer.get("mlp"))
        if s.kv_heads < 1 or s.heads % s.kv_heads or s.window < 0 or s.keep_first < 0 or s.softcap < 0 or taps < 0 or (mask and s.window < 1):
            raise ValueError(f"Gulazen layer {i}: inconsistent geometry")
        mixers.append(s)
    first, routed = mixers[0], [s.moe for s in mixers if s.moe is not None]
    return cls(model_type="gulazen", vocab_size=int(d["vocab"]), hidden_size=width,
               intermediate_size=max([s.ff for s in mixers] + [m.moe_intermediate_size for m in routed]), num_hidden_layers=len(mixers),
               num_attention_heads=first.heads, num_key_value_heads=first.kv_heads, head_dim=first.dim, rms_norm_eps=float(d["norm"]["eps"]),
               max_position_embeddings=int(d.get("max_position_embeddings", 1 << 20)), tie_word_embeddings=True,
               layer_types=[s.kind for s in mixers], eos_token_id=d.get("eos_token_id"), bos_token_id=d.get("bos_token_id"),
               torch_dtype=str(d.get("torch_dtype", "bfloat16")), mixers=mixers)


def config_dict(cfg) -> dict:
    """ModelConfig -> ``config.json`` (inverse of :func:`config_from_dict`)."""
    layers = []
    for s in cfg.mixers:
        m = {"heads": s.heads, "kv_heads": s.kv_heads, "dim": s.dim, "vdim": s.vdim, "scale": s.scale}
        if s.softcap:
            m["softcap"] = s.softcap
        if s.window:
            m["mask"] = {"size": s.window, "keep_first": s.keep_first}
        mlp = {"kind": "dense", "ff": s.ff} if s.ff else None
        if s.moe is not None:
            mlp = {"kind": "moe", "expert": {"ff": s.moe.moe_intermediate_size},
                   "router": {"experts": s.moe.num_experts, "top": s.moe.num_experts_per_tok}}
            if s.moe.shared_ff:
                mlp["shared"] = {"ff": s.moe.shared_ff}
        layers.append({"type": s.kind, "mixer": m, "mlp": mlp})
    d = {"architecture": "Gulazen", "vocab": cfg.vocab_size, "width": cfg.hidden_size, "norm": {"eps": cfg.rms_norm_eps}, "layers": layers}
    if cfg.mixers[0].lead_conv:
        d["canon"] = {"taps": cfg.mixers[0].lead_conv}
    for k in ("eos_token_id", "bos_token_id"):
        if getattr(cfg, k) is not None:
            d[k] = getattr(cfg, k)
    return d


# ---------------------------------------------------------------------------------------------- tensors
def canonical_access(get, has):
    """The tensors outside the layers under the names the generic loader asks for (the head is the embedding)."""
    def resolve(name):
        alt = TOP_LEVEL.get(name)
        return alt if alt is not None and has(alt) else name

    return (lambda name: get(resolve(name))), (lambda name: has(resolve(name)))


def tensor_shapes(cfg) -> dict:
    """Every tensor of a checkpoint of this geometry: name -> shape."""
    W = cfg.hidden_size
    out = {"embed": (cfg.vocab_size, W), "final.norm": (W,)}

    def gated(p, ff):
        out.update({p + ".gate": (ff, W), p + ".up": (ff, W), p + ".down": (W, ff)})

    for i, s in enumerate(cfg.mixers):
        p, q, k, v = f"l{i}.mix.", s.heads * s.dim, s.kv_heads * s.dim, s.kv_heads * s.vdim
        out.update({f"l{i}.norm1": (W,), f"l{i}.ls1": (W,), p + "q": (q, W), p + "k": (k, W), p + "v": (v, W), p + "q.norm": (q,),
                    p + "k.norm": (k,), p + "talk": (s.heads, s.heads), p + "sink": (s.heads,), p + "o": (W, s.heads * s.vdim)})
        if s.lead_conv:
            out[f"l{i}.canon1"] = (W, s.lead_conv)
        if s.ff or s.moe is not None:
            out.update({f"l{i}.norm2": (W,), f"l{i}.ls2": (W,)})
        p = f"l{i}.mlp."
        if s.ff:
            out.update({p + "up": (s.ff, W), p + "down": (W, s.ff), p + "act": (2,)})
        if s.moe is not None:
            out.update({p + "router": (s.moe.num_experts, W), p + "router.b": (s.moe.num_experts,)})
            for e in range(s.moe.num_experts):
                gated(f"{p}e{e}", s.moe.moe_intermediate_size)
            if s.moe.shared_ff:
                gated(p + "shared", s.moe.shared_ff)
    return out


def random_tensor(name: str, shape: tuple, generator, std: float = 0.02, device="cpu") -> torch.Tensor:
    """Seeded fp32 values of one tensor: norms and layer scales of one, heads mixed around the identity, convolutions that add something
    of their input's size, N(0, std) otherwise."""
    last = name.rsplit(".", 1)[-1]
    if name.endswith((".q.norm", ".k.norm")) or last in ("ls1", "ls2"):
        return torch.ones(shape, dtype=torch.float32, device=device)
    if "norm" in last:
        return torch.zeros(shape, dtype=torch.float32, device=device)
    t = torch.randn(shape, generator=generator, dtype=torch.float32, device=device)
    if last == "talk":
        return torch.eye(shape[0], device=device) + t * (0.3 * shape[0] ** -0.5)
    if last == "canon1":
        return t * (0.3 * shape[1] ** -0.5)
    return t * std


def build(model, cfg, get, has, up) -> None:
    """Fill ``model.layers`` (called by the generic loader after the embedding, final norm and head)."""
    from .llama import LayerWeights
    from .moe import expert_block

    f32 = lambda n: up(get(n), torch.float32)                                          # noqa: E731
    pad = torch.nn.functional.pad
    model.position_freq = base_inv_freq(POSITION_BASE, cfg.hidden_size).to(device=model.device, dtype=torch.float32)
    if model.final_norm is not None:
        model.final_norm = 1.0 + model.final_norm
    for li, s in enumerate(cfg.mixers):
        p, q = f"l{li}.mix.", f"l{li}.mlp."
        lw = LayerWeights(attn_norm=(1.0 + f32(f"l{li}.norm1")) * f32(f"l{li}.ls1"), wqkv=None, wo=up(get(p + "o")), ffn_norm=None)
        lw.block_kind = "gulazen"
        mats = [get(p + n) for n in "qkv"]                # zero rows bring rows of the product to whole 16-byte pieces
        lw.wqkv = up(pad(torch.cat(mats), (0, 0, 0, -sum(m.shape[0] for m in mats) % 8)))
        lw.q_norm, lw.k_norm, lw.sinks = f32(p + "q.norm"), f32(p + "k.norm"), f32(p + "sink")
        e = lw.extra = {"talk": up(get(p + "talk"))}
        if s.lead_conv:
            e["taps"] = up(get(f"l{li}.canon1").t(), torch.float32)
        if s.ff or s.moe is not None:
            lw.ffn_norm = (1.0 + f32(f"l{li}.norm2")) * f32(f"l{li}.ls2")
        if s.ff:
            n = -s.ff % 8
            lw.w_gate_up, lw.w_down = up(pad(get(q + "up"), (0, 0, 0, n))), up(pad(get(q + "down"), (0, n)))
            e["act"] = ops.XIELU.from_checkpoint(*get(q + "act").float().tolist())
        if s.moe is not None:
            lw.moe = expert_block(s.moe, li, q, get, up)
            lw.moe.router_linear_bias = up(get(q + "router.b")) if has(q + "router.b") else None
        model.layers.append(lw)


# ---------------------------------------------------------------------------------------------- forward
def enter(model, batch):
    """Embedding and position vectors: the start of the fp32 stream."""
    return ops.embedding_stream(batch.token_ids, model.embed, want_act=False, positions=batch.positions, inv_freq=model.position_freq)[0]


def _lead(model, li, batch, kv):
    """The convolution in front of a layer's mixer as the operators take it (None: the layer has none)."""
    i = li - model.first_layer
    taps = model.layers[i].extra.get("taps") if i < len(model.layers) else None
    return None if taps is None else ops.StreamConv(taps, kv.layer_state.get(li), batch, kv.page_to_slot)


def block_forward(model, li, lw, x, batch, kv):
    s, eps = model.cfg.mixers[li], model.cfg.rms_norm_eps
    if batch.stream is not None and batch.stream[0] is x:
        h = batch.stream[1]                               # the kernel that finished the previous layer has convolved it
    else:
        lead = _lead(model, li, batch, kv)
        h = ops.stream_conv(x, lead, model.dtype) if lead is not None else x.to(model.dtype)
    # Decode steps continue with the next layer's convolution at once. It moves that layer's state on, so it is left to the layer itself
    # where somebody may replace the stream in between.
    lead = _lead(model, li + 1, batch, kv) if not batch.is_prefill and batch.q_per_seq == 1 and model.observer is None else None
    y, weight, routed = _attention(model, li, lw, s, h, batch, kv), lw.attn_norm, None
    if s.ff or s.moe is not None:
        x, act = ops.rms_residual(y, weight, eps, residual=x, act_dtype=model.dtype)
        y, routed = _feed(model, lw, s, act)
        weight = lw.ffn_norm
    x, h = ops.rms_residual(y, weight, eps, residual=x, act_dtype=model.dtype, routed=routed, conv=lead, want_act=lead is not None)
    batch.stream = (x, h) if lead is not None else None
    return x


def _feed(model, lw, s, act):
    """(output in the compute dtype or None, expert rows still to be added or None)"""
    if s.ff:
        return ops.linear(ops.linear(act, lw.w_gate_up, activation=lw.extra["act"]), lw.w_down), None
    if model.observer is not None:
        return lw.moe.observed_call(act, None, model.observer), None
    logits = lw.moe.router_logits(act)
    return lw.moe.shared_out(act), lw.moe.routed_rows(act, logits)


def final_norm(model, x):
    """The normalised rows the output head reads."""
    return ops.rms_residual(x, model.final_norm, model.cfg.rms_norm_eps, act_dtype=model.dtype)[1]


def _attention(model, li, lw, s, h, batch, kv):
    qkv = ops.linear(h, lw.wqkv)
    k_cache, v_cache = kv.layer(li)
    q = ops.qkv_prepare(qkv, batch.positions, batch.slots, model.position_freq[:0], k_cache, v_cache, s.heads, s.kv_heads, s.dim, s.vdim,
                        lw.q_norm, lw.k_norm, model.cfg.rms_norm_eps)
    attn = ops.talking_attention(q, k_cache, v_cache, batch, lw.extra["talk"], s.scale, s.softcap, lw.sinks, s.window, s.keep_first)
    return ops.linear(attn.view(attn.shape[0], -1), lw.wo)
