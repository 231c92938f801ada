"""Lenitar: a decoder with one LayerNorm per layer whose output feeds both sublayers - a mixer (latent attention or the mLSTM
matrix memory, with sizes of its own) and a group-routed mixture of experts - and both are added to the stream at once:
``x <- x + mixer(h) + experts(h)``, ``h = norm(x)``.

The stream is fp32. One kernel (:func:`ops.residual_norm`) adds a layer's mixer and the weighted rows of its experts and
normalises the sum for the next layer, so a layer starts from the activations its predecessor left in ``batch.stream``.
Projections of ``h`` are fused at load; those that stay fp32 (router, recurrence gates) form a second, small one:

* latent attention: ``[gate | query latent | latent, rotated key part]`` -> norms, rotation and the append of one row per token
  (:func:`ops.latent_prepare`) -> queries -> attention over the cached rows (:func:`ops.latent_attention`: decode in latent
  space, long portions over keys and values expanded from it; sliding window, sinks, output gate) -> output projection;
* mlstm: ``[q | k | v | gate]`` and the fp32 gates -> recurrence, per-head norm, output gate (:func:`ops.mlstm`) -> output
  projection.

Runs in bf16 and, everything in true 32-bit, in fp32.
"""
from __future__ import annotations

import torch

from .. import ops
from .rope import base_inv_freq

TOP_LEVEL = {"model.embed_tokens.weight": "embed", "model.norm.weight": "final.norm", "lm_head.weight": "head"}


# ---------------------------------------------------------------------------------------------- configuration
def _routed(i: int, mlp):
    from .config import RoutedSpec

    if mlp is None:
        return None
    if mlp.get("kind") != "moe":
        raise ValueError(f"Lenitar layer {i}: unknown feed-forward {mlp.get('kind')!r}")
    r = mlp["router"]
    g = r.get("groups") or {}
    spec = RoutedSpec(int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"]), int(g.get("count", 1)), int(g.get("keep", 1)))
    per = spec.num_experts // max(1, spec.n_group)
    if (spec.n_group < 1 or spec.num_experts % spec.n_group or not 1 <= spec.topk_group <= spec.n_group
            or not 1 <= spec.num_experts_per_tok <= spec.topk_group * per):
        raise ValueError(f"Lenitar layer {i}: inconsistent expert groups")
    return spec


def config_from_dict(cls, d: dict):
    """``config.json`` -> ModelConfig: the layer list becomes ``mixers``, the generic fields describe the whole."""
    from .config import MixerSpec

    mixers = []
    for i, layer in enumerate(d["layers"]):
        kind, m = layer["type"], layer["mixer"]
        if kind not in ("latent_attention", "mlstm"):
            raise ValueError(f"Lenitar layer {i}: unknown mixer {kind!r}")
        s = MixerSpec(kind, heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), moe=_routed(i, layer.get("mlp")))
        if kind == "mlstm":
            s.gate_cap = float(m["gate_cap"])
        else:
            s.q_rank, s.kv_rank, s.rot_dims = int(m["q_rank"]), int(m["kv_rank"]), int(m["rot_dim"])
            s.scale, s.rot_base = float(m["scale"]), float(m["rot"]["base"])
            s.window = int((m.get("mask") or {}).get("size", 0))
            if int(m["rot"].get("dims", s.rot_dims)) != s.rot_dims or s.rot_dims % 2 or s.window < 0:
                raise ValueError(f"Lenitar layer {i}: inconsistent attention geometry")
        mixers.append(s)
    attn = [s for s in mixers if s.kind == "latent_attention"] or [MixerSpec("latent_attention", 1, dim=64, vdim=64)]
    routed = [s.moe for s in mixers if s.moe is not None]
    return cls(model_type="lenitar", vocab_size=int(d["vocab"]), hidden_size=int(d["width"]),
               intermediate_size=max([m.moe_intermediate_size for m in routed], default=0), num_hidden_layers=len(mixers),
               num_attention_heads=attn[0].heads, num_key_value_heads=1, head_dim=attn[0].dim + attn[0].rot_dims,
               rms_norm_eps=float(d["norm"]["eps"]), rope_theta=attn[0].rot_base,
               max_position_embeddings=int(d.get("max_position_embeddings", 1 << 20)), tie_word_embeddings=False,
               embedding_scale=float(d["embedding"]["scale"]), layer_types=[s.kind for s in mixers],
               eos_token_id=d.get("eos_token_id"), bos_token_id=d.get("bos_token_id"),
               torch_dtype=str(d.get("torch_dtype", "bfloat16")), mixers=mixers)


def config_dict(cfg) -> dict:
    """ModelConfig -> ``config.json`` (inverse of :func:`config_from_dict`)."""
    layers = []
    for s in cfg.mixers:
        m = {"heads": s.heads, "dim": s.dim, "vdim": s.vdim}
        if s.kind == "mlstm":
            m["gate_cap"] = s.gate_cap
        else:
            m.update(rot_dim=s.rot_dims, q_rank=s.q_rank, kv_rank=s.kv_rank, scale=s.scale, rot={"dims": s.rot_dims, "base": s.rot_base})
            if s.window:
                m["mask"] = {"size": s.window}
        mlp = None
        if s.moe is not None:
            mlp = {"kind": "moe", "expert": {"ff": s.moe.moe_intermediate_size},
                   "router": {"experts": s.moe.num_experts, "top": s.moe.num_experts_per_tok,
                              "groups": {"count": s.moe.n_group, "keep": s.moe.topk_group}}}
        layers.append({"type": s.kind, "mixer": m, "mlp": mlp})
    d = {"architecture": "Lenitar", "vocab": cfg.vocab_size, "width": cfg.hidden_size, "norm": {"eps": cfg.rms_norm_eps},
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


def tensor_shapes(cfg) -> dict:
    """Every tensor of a checkpoint of this geometry: name -> shape."""
    W = cfg.hidden_size
    out = {"embed": (cfg.vocab_size, W), "head": (cfg.vocab_size, W), "final.norm": (W,), "final.norm.b": (W,)}
    for i, s in enumerate(cfg.mixers):
        p, v = f"l{i}.mix.", s.heads * s.vdim
        out.update({f"l{i}.norm1": (W,), f"l{i}.norm1.b": (W,), p + "g": (v, W), p + "o": (W, v)})
        if s.kind == "mlstm":
            qk = s.heads * s.dim
            out.update({p + "q": (qk, W), p + "k": (qk, W), p + "v": (v, W), p + "norm": (v,)})
            for n in "if":
                out.update({p + n: (s.heads, W), p + n + ".b": (s.heads,)})
        else:
            out.update({p + "dq": (s.q_rank, W), p + "dq.norm": (s.q_rank,), p + "uq": (s.heads * (s.dim + s.rot_dims), s.q_rank),
                        p + "dkv": (s.kv_rank + s.rot_dims, W), p + "dkv.norm": (s.kv_rank,), p + "uk": (s.heads * s.dim, s.kv_rank),
                        p + "uv": (v, s.kv_rank), p + "sink": (s.heads,)})
        if s.moe is not None:
            q, ff = f"l{i}.mlp.", s.moe.moe_intermediate_size
            out[q + "router"] = (s.moe.num_experts, W)
            for e in range(s.moe.num_experts):
                out.update({f"{q}e{e}.gate": (ff, W), f"{q}e{e}.up": (ff, W), f"{q}e{e}.down": (W, ff)})
    return out


def random_tensor(name: str, shape: tuple, generator, std: float = 0.02, device="cpu") -> torch.Tensor:
    """Seeded fp32 values of one tensor: unit norms, open forget gates, N(0, std) otherwise."""
    if name.endswith("norm") or name.endswith("norm1"):
        return torch.ones(shape, dtype=torch.float32, device=device)
    t = torch.randn(shape, generator=generator, dtype=torch.float32, device=device) * std
    return t + 4.0 if name.endswith(".f.b") else t


def build(model, cfg, get, has, up) -> None:
    """Fill ``model.layers`` (called by the generic loader after the embedding, final norm and head)."""
    from .llama import LayerWeights
    from .moe import expert_block

    f32 = lambda n: up(get(n), torch.float32)                                          # noqa: E731

    def fused(names, pad: int = 1):
        """Rows of several projections of the same input as one matrix; ``pad``: zero rows up to a multiple of this."""
        w = torch.cat([get(n) for n in names], 0)
        return up(torch.nn.functional.pad(w, (0, 0, 0, -w.shape[0] % pad)))

    model.final_norm_b = f32("final.norm.b")
    for li, s in enumerate(cfg.mixers):
        p = f"l{li}.mix."
        lw = LayerWeights(attn_norm=f32(f"l{li}.norm1"), wqkv=None, wo=up(get(p + "o")), ffn_norm=None)
        lw.block_kind = "lenitar"
        e = lw.extra = {"norm_b": f32(f"l{li}.norm1.b")}
        small = []                                        # projections whose results stay fp32: gates of the recurrence, router
        if s.kind == "mlstm":
            lw.wqkv = fused([p + n for n in "qkvg"], pad=8)
            e["o_norm"] = f32(p + "norm")
            small = [p + "i", p + "f"]
        else:
            lw.wqkv = fused([p + n for n in ("g", "dq", "dkv")], pad=8)
            lw.mla_q_norm, lw.mla_kv_norm, lw.mla_q_b = f32(p + "dq.norm"), f32(p + "dkv.norm"), up(get(p + "uq"))
            lw.sinks = f32(p + "sink")
            e["kv_up"] = fused([p + "uk", p + "uv"])                                    # [H dim | H vdim, kv_rank]
            keys = s.heads * s.dim
            lw.mla_w_uv = e["kv_up"][keys:].view(s.heads, s.vdim, s.kv_rank)
            # the absorbed form multiplies queries by the transpose
            lw.mla_w_uk = e["kv_up"][:keys].view(s.heads, s.dim, s.kv_rank).transpose(1, 2).contiguous()
            e["inv_freq"] = base_inv_freq(s.rot_base, s.rot_dims).to(device=model.device, dtype=torch.float32)
        if s.moe is not None:
            small.append(f"l{li}.mlp.router")
            lw.moe = expert_block(s.moe, li, f"l{li}.mlp.", get, up)
        if small:
            e["small"] = fused(small)
            bias = [get(n + ".b") if has(n + ".b") else torch.zeros(get(n).shape[0]) for n in small]
            e["small_b"] = up(torch.cat([b.to(e["small"].device, torch.float32) for b in bias])) if any(has(n + ".b") for n in small) else None
        model.layers.append(lw)


# ---------------------------------------------------------------------------------------------- forward
def _norm(model, i: int):
    """Weight and bias of the norm in front of layer i (of this shard's list), None behind the last one."""
    if i >= len(model.layers):
        return None, None
    return model.layers[i].attn_norm, model.layers[i].extra["norm_b"]


def enter(model, batch):
    """The scaled embedding as the start of the fp32 stream, and the first layer's input."""
    x = ops.embedding_stream(batch.token_ids, model.embed, scale=model.cfg.embedding_scale, want_act=False)[0]
    batch.stream = (x, _normed(model, 0, x))
    return x


def _normed(model, i: int, x):
    weight, bias = _norm(model, i)
    return ops.residual_norm(x, weight=weight, bias=bias, eps=model.cfg.rms_norm_eps, act_dtype=model.dtype)[1]


def block_forward(model, li, lw, x, batch, kv):
    s, i = model.cfg.mixers[li], li - model.first_layer
    # the activations the previous layer left, unless somebody replaced the stream
    h = batch.stream[1] if batch.stream is not None and batch.stream[0] is x else _normed(model, i, x)
    e = lw.extra
    small = ops.linear(h, e["small"], bias=e["small_b"], out_dtype=torch.float32) if "small" in e else None
    routed = None
    if s.moe is not None:
        logits = small[:, small.shape[1] - s.moe.num_experts:]
        if model.observer is not None:
            x = x + lw.moe.observed_call(h, None, model.observer).float()
        else:
            routed = lw.moe.routed_rows(h, logits)
    y = _mlstm(model, li, lw, s, h, small, batch, kv) if s.kind == "mlstm" else _latent_attention(model, li, lw, s, h, batch, kv)
    weight, bias = _norm(model, i + 1)
    batch.stream = ops.residual_norm(x, y, routed, weight=weight, bias=bias, eps=model.cfg.rms_norm_eps, act_dtype=model.dtype)
    return batch.stream[0]


def final_norm(model, x):
    """The normalised rows the output head reads."""
    return ops.residual_norm(x, weight=model.final_norm, bias=model.final_norm_b, eps=model.cfg.rms_norm_eps, act_dtype=model.dtype)[1]


def _latent_attention(model, li, lw, s, h, batch, kv):
    proj = ops.linear(h, lw.wqkv)
    gates = s.heads * s.vdim
    cache, _ = kv.layer(li)
    e = lw.extra
    cq = ops.latent_prepare(proj[:, gates:], s.q_rank, s.kv_rank, s.rot_dims, lw.mla_q_norm, lw.mla_kv_norm, model.cfg.rms_norm_eps,
                            batch.positions, batch.slots, e["inv_freq"], cache)
    q = ops.linear(cq, lw.mla_q_b)
    y = ops.latent_attention(q, cache, batch, lw.mla_w_uk, lw.mla_w_uv, e["kv_up"], proj[:, :gates], lw.sinks, e["inv_freq"],
                             s.heads, s.dim, s.rot_dims, s.scale, s.window)
    return ops.linear(y, lw.wo)


def _mlstm(model, li, lw, s, h, small, batch, kv):
    proj = ops.linear(h, lw.wqkv)
    y = ops.mlstm(proj, small[:, :2 * s.heads], lw.extra["o_norm"], kv.layer_state[li], s.heads, s.dim, s.vdim, s.gate_cap,
                  model.cfg.rms_norm_eps, batch, kv.page_to_slot)
    return ops.linear(y, lw.wo)
