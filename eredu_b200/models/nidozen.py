"""Nidozen: a decoder whose layers each name their mixer - softmax attention over chunks of positions, gated linear
attention or the minGRU recurrence - with sizes of their own, and an optional squared-ReLU feed-forward.

A sublayer reads the residual stream as it is; its output goes through an RMSNorm with one learned number before it is
added: ``x <- x + g * rms(mixer(x))``, then ``x <- x + g' * rms(ff(x))``. The stream is kept in fp32 together with its copy
in the compute dtype, which is what the projections read; one kernel (:func:`ops.rms_residual`) normalises, adds and writes
both. Projections that read the same input are fused at load:

* attention: ``[q | k | v]`` -> norm over the whole q and the whole k, partial rotation, per-head value norm and the append
  to the pages (:func:`ops.qkv_prepare`; decode steps do this inside the attention kernel) -> paged attention whose queries
  see the keys of their own chunk -> output projection. A layer with ``kv_from`` projects queries only and reads the pages
  of that layer;
* gla: ``[q | k | v | gate | low-rank decay]`` -> decay, recurrence, per-head norm and gate (:func:`ops.gla_attention`);
* mingru: ``[z | x | gate]`` -> gates, recurrence and output gate (:func:`ops.mingru_scan`).

Recurrent states are fp32, one slot per sequence and a tensor per layer (:meth:`PagedKVCache.enable_layer_states`).
Runs in bf16 and, everything in true 32-bit, in fp32.
"""
from __future__ import annotations

import torch

from .. import ops
from .rope import base_inv_freq

TOP_LEVEL = {"model.embed_tokens.weight": "embed", "model.norm.weight": "final.norm", "lm_head.weight": "head"}
DEFAULT_DECAY_RANK = 16      # rank of the decay projection in randomly initialised models (checkpoints: the tensor's own)


# ---------------------------------------------------------------------------------------------- configuration
def config_from_dict(cls, d: dict):
    """``config.json`` -> ModelConfig: the layer list becomes ``mixers``, the generic fields describe the whole."""
    from .config import MixerSpec

    mixers = []
    for i, layer in enumerate(d["layers"]):
        kind, m, mlp = layer["type"], layer.get("mixer") or {}, layer.get("mlp")
        if kind not in ("attention", "gla", "mingru"):
            raise ValueError(f"Nidozen layer {i}: unknown mixer {kind!r}")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"Nidozen layer {i}: unknown feed-forward {mlp.get('kind')!r}")
        s = MixerSpec(kind, ff=int(mlp["ff"]) if mlp is not None else 0)
        if kind == "mingru":
            s.width = int(m["width"])
        else:
            s.heads, s.dim, s.vdim = int(m["heads"]), int(m["dim"]), int(m["vdim"])
        if kind == "gla":
            s.tau = float(m["tau"])
        if kind == "attention":
            s.kv_heads, s.scale = int(m["kv_heads"]), float(m["scale"])
            s.chunk = int((m.get("mask") or {}).get("size", 0))
            rot = m.get("rot") or {}
            s.rot_dims, s.rot_base = int(rot.get("dims", 0)), float(rot.get("base", 10000.0))
            s.kv_from = int(m["kv_from"]) if m.get("kv_from") is not None else None
            if s.heads % s.kv_heads or s.rot_dims % 2 or s.rot_dims > s.dim or s.chunk < 0:
                raise ValueError(f"Nidozen layer {i}: inconsistent attention geometry")
            if s.kv_from is not None:
                donor = mixers[s.kv_from] if 0 <= s.kv_from < i else None
                if donor is None or donor.kind != "attention" or donor.kv_from is not None or \
                        (donor.kv_heads, donor.dim, donor.vdim) != (s.kv_heads, s.dim, s.vdim):
                    raise ValueError(f"Nidozen layer {i}: layer {s.kv_from} has no keys and values it could read")
        mixers.append(s)
    attn = [s for s in mixers if s.kind == "attention"] or [MixerSpec("attention", 1, 1, 64, 64)]
    cfg = cls(model_type="nidozen", vocab_size=int(d["vocab"]), hidden_size=int(d["width"]),
              intermediate_size=max(s.ff for s in mixers), num_hidden_layers=len(mixers), num_attention_heads=attn[0].heads,
              num_key_value_heads=attn[0].kv_heads, head_dim=attn[0].dim, rms_norm_eps=float(d["norm"]["eps"]),
              rope_theta=attn[0].rot_base, max_position_embeddings=int(d.get("max_position_embeddings", 1 << 20)),
              tie_word_embeddings=False, layer_types=[s.kind for s in mixers], eos_token_id=d.get("eos_token_id"),
              bos_token_id=d.get("bos_token_id"), torch_dtype=str(d.get("torch_dtype", "bfloat16")), mixers=mixers)
    return cfg


def config_dict(cfg) -> dict:
    """ModelConfig -> ``config.json`` (inverse of :func:`config_from_dict`)."""
    layers = []
    for s in cfg.mixers:
        if s.kind == "mingru":
            m = {"width": s.width}
        elif s.kind == "gla":
            m = {"heads": s.heads, "dim": s.dim, "vdim": s.vdim, "tau": s.tau}
        else:
            m = {"heads": s.heads, "kv_heads": s.kv_heads, "dim": s.dim, "vdim": s.vdim, "scale": s.scale}
            if s.chunk:
                m["mask"] = {"size": s.chunk}
            if s.rot_dims:
                m["rot"] = {"dims": s.rot_dims, "base": s.rot_base}
            if s.kv_from is not None:
                m["kv_from"] = s.kv_from
        layers.append({"type": s.kind, "mixer": m, "mlp": {"kind": "dense", "ff": s.ff} if s.ff else None})
    d = {"architecture": "Nidozen", "vocab": cfg.vocab_size, "width": cfg.hidden_size, "norm": {"eps": cfg.rms_norm_eps},
         "layers": layers}
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
    out = {"embed": (cfg.vocab_size, W), "head": (cfg.vocab_size, W), "final.norm": ()}
    for i, s in enumerate(cfg.mixers):
        p = f"l{i}.mix."
        out[f"l{i}.norm1"] = ()
        if s.kind == "mingru":
            out.update({p + "z": (s.width, W), p + "z.b": (s.width,), p + "x": (s.width, W), p + "x.b": (s.width,),
                        p + "g": (s.width, W), p + "o": (W, s.width)})
        elif s.kind == "gla":
            qk, v = s.heads * s.dim, s.heads * s.vdim
            out.update({p + "q": (qk, W), p + "k": (qk, W), p + "v": (v, W), p + "g": (v, W), p + "o": (W, v),
                        p + "norm": (s.vdim,), p + "a1": (decay_rank, W), p + "a2": (qk, decay_rank), p + "a2.b": (qk,)})
        else:
            q, k, v = s.heads * s.dim, s.kv_heads * s.dim, s.kv_heads * s.vdim
            out.update({p + "q": (q, W), p + "q.b": (q,), p + "q.norm": (q,), p + "o": (W, s.heads * s.vdim), p + "o.b": (W,)})
            if s.kv_from is None:
                out.update({p + "k": (k, W), p + "k.b": (k,), p + "k.norm": (k,), p + "v": (v, W), p + "v.b": (v,)})
        if s.ff:
            out.update({f"l{i}.norm2": (), f"l{i}.mlp.up": (s.ff, W), f"l{i}.mlp.down": (W, s.ff)})
    return out


def random_tensor(name: str, shape: tuple, generator, std: float = 0.02, device="cpu") -> torch.Tensor:
    """Seeded fp32 values of one tensor: unit norms, N(0, std) matrices and biases."""
    if name.endswith("norm") or ".norm" in name:
        return torch.ones(shape, dtype=torch.float32, device=device)
    return torch.randn(shape, generator=generator, dtype=torch.float32, device=device) * std


def build(model, cfg, get, has, up) -> None:
    """Fill ``model.layers`` (called by the generic loader after the embedding, final norm and head)."""
    from .llama import LayerWeights

    model.final_norm = model.final_norm.reshape(1)
    f32 = lambda n: up(get(n), torch.float32)                                          # noqa: E731
    opt = lambda n: get(n) if has(n) else None                                         # noqa: E731

    def fused(names, pad: int = 1):
        """Rows of several projections of the same input as one matrix, with their biases (zero where there is none);
        ``pad``: zero rows bring the last projection to a multiple of this."""
        mats, biases = [get(n) for n in names], [opt(n + ".b") for n in names]
        mats[-1] = torch.nn.functional.pad(mats[-1], (0, 0, 0, -mats[-1].shape[0] % pad))
        bias = None
        if any(b is not None for b in biases):
            bias = up(torch.cat([b if b is not None else torch.zeros(m.shape[0], dtype=m.dtype, device=m.device) for m, b in zip(mats, biases)]))
        return up(torch.cat(mats, 0)), bias

    for li, s in enumerate(cfg.mixers):
        p = f"l{li}.mix."
        lw = LayerWeights(attn_norm=f32(f"l{li}.norm1").reshape(1), wqkv=None, wo=up(get(p + "o")), ffn_norm=None)
        lw.block_kind = "nidozen"
        lw.bo = up(get(p + "o.b")) if has(p + "o.b") else None
        if s.kind == "attention":
            own = s.kv_from is None
            lw.wqkv, lw.bqkv = fused([p + n for n in ("qkv" if own else "q")])
            lw.q_norm = f32(p + "q.norm")
            lw.k_norm = f32(p + "k.norm") if own else None
            inv = base_inv_freq(s.rot_base, s.rot_dims) if s.rot_dims else torch.zeros(0)
            lw.extra = {"inv_freq": inv.to(device=model.device, dtype=torch.float32)}
        elif s.kind == "gla":
            # the rank of the decay projection is padded to a multiple of 8 with zeros: rows of the fused projection are then
            # a whole number of 16-byte pieces
            lw.wqkv, lw.bqkv = fused([p + n for n in ("q", "k", "v", "g", "a1")], pad=8)
            a2 = f32(p + "a2")
            lw.extra = {"a2": torch.nn.functional.pad(a2, (0, -a2.shape[1] % 8)).contiguous(), "a2_b": f32(p + "a2.b"),
                        "o_norm": f32(p + "norm")}
        else:
            lw.wqkv, lw.bqkv = fused([p + n for n in "zxg"])
        if s.ff:
            lw.ffn_norm = f32(f"l{li}.norm2").reshape(1)
            lw.w_gate_up, lw.w_down = up(get(f"l{li}.mlp.up")), up(get(f"l{li}.mlp.down"))
        model.layers.append(lw)


# ---------------------------------------------------------------------------------------------- forward
def enter(model, batch):
    """The embedding as the start of the fp32 residual stream (and its compute-dtype copy)."""
    x, act = ops.embedding_stream(batch.token_ids, model.embed)
    batch.stream = (x, act)
    return x


def _act(model, x, batch):
    """Compute-dtype copy of the residual stream: what the previous sublayer left, unless somebody replaced the stream."""
    if batch.stream is not None and batch.stream[0] is x:
        return batch.stream[1]
    return x.to(model.dtype)


def block_forward(model, li, lw, x, batch, kv):
    s, eps = model.cfg.mixers[li], model.cfg.rms_norm_eps
    act = _act(model, x, batch)
    y = _MIXERS[s.kind](model, li, lw, s, act, batch, kv)
    x, act = ops.rms_residual(y, lw.attn_norm, eps, residual=x, act_dtype=model.dtype)
    if s.ff:
        a = ops.linear(act, lw.w_gate_up, activation="relu2")
        x, act = ops.rms_residual(ops.linear(a, lw.w_down), lw.ffn_norm, eps, residual=x, act_dtype=model.dtype)
    batch.stream = (x, act)
    return x


def final_norm(model, x):
    """The normalised rows the output head reads."""
    _, act = ops.rms_residual(x, model.final_norm, model.cfg.rms_norm_eps, act_dtype=model.dtype)
    return act


def _attention(model, li, lw, s, act, batch, kv):
    qkv = ops.linear(act, lw.wqkv, bias=lw.bqkv)
    k_cache, v_cache = kv.layer(li)
    eps, inv_freq, own = model.cfg.rms_norm_eps, lw.extra["inv_freq"], s.kv_from is None
    if batch.is_prefill:
        q = ops.qkv_prepare(qkv, batch.positions, batch.slots, inv_freq, k_cache, v_cache, s.heads, s.kv_heads, s.dim, s.vdim,
                            lw.q_norm, lw.k_norm, eps, value_norm=True, append=own)
        attn = ops.attention_prefill(q, k_cache, v_cache, batch.block_table, batch.seq_lens, batch.cu_q, batch.max_q_len,
                                     s.scale, chunk=s.chunk)
    else:
        attn = ops.attention_decode_rope(qkv, k_cache, v_cache, batch.block_table, batch.seq_lens, batch.q_per_seq, s.scale,
                                         batch.positions, batch.slots, inv_freq, s.heads, s.kv_heads, s.dim, q_norm_w=lw.q_norm,
                                         k_norm_w=lw.k_norm, norm_eps=eps, splits=batch.layer_splits(s.kv_heads, s.chunk),
                                         chunk=s.chunk, value_dim=s.vdim, norm_whole=True, value_norm=True, append=own)
    return ops.linear(attn.view(attn.shape[0], -1), lw.wo, bias=lw.bo)


def _gla(model, li, lw, s, act, batch, kv):
    proj = ops.linear(act, lw.wqkv, bias=lw.bqkv)
    e = lw.extra
    y = ops.gla_attention(proj, e["a2"], e["a2_b"], e["o_norm"], kv.layer_state[li], s.heads, s.dim, s.vdim, s.tau,
                          model.cfg.rms_norm_eps, batch, kv.page_to_slot)
    return ops.linear(y, lw.wo)


def _mingru(model, li, lw, s, act, batch, kv):
    proj = ops.linear(act, lw.wqkv, bias=lw.bqkv)
    y = ops.mingru_scan(proj, kv.layer_state[li], s.width, batch, kv.page_to_slot)
    return ops.linear(y, lw.wo)


_MIXERS = {"attention": _attention, "gla": _gla, "mingru": _mingru}
