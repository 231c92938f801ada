"""Plain whole-sequence restatement of the Gulazen decoder: one function per mechanism, dense masked scores, expert by expert. The
oracle of the Gulazen tests; it shares nothing with the package. ``cfg`` is the parsed config.json, ``w`` maps tensor names to tensors;
everything runs in ``dtype``."""
import math

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_plus_one(x, weight, eps):
    """RMS norm whose stored weight is the distance from one."""
    return unit_rms(x, eps) * (1.0 + weight.to(x.dtype))


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + x.clamp_min(0)


def soft_cap(x, cap):
    return cap * torch.tanh(x / cap)


def xielu(x, p, q):
    """softplus(p) x^2 + x / 2 above zero; (1/2 + softplus(q)) (e^x - 1 - x) + x / 2 below."""
    below = (0.5 + softplus(q)) * (torch.expm1(x.clamp_max(0)) - x.clamp_max(0))
    return torch.where(x > 0, softplus(p) * x * x, below) + x / 2


def position_vectors(positions, width, dtype):
    """[T, width]: sin and cos of position * 10000^(-2 i / width) side by side."""
    out = torch.zeros(len(positions), width, dtype=torch.float64)
    for i in range((width + 1) // 2):
        a = positions.to(torch.float64) * 10000.0 ** (-2.0 * i / width)
        out[:, 2 * i] = torch.sin(a)
        if 2 * i + 1 < width:
            out[:, 2 * i + 1] = torch.cos(a)
    return out.to(dtype)


def causal_conv(x, taps):
    """x [T, C], taps [C, K]: the tap K - 1 multiplies the position itself, the one before it the position before, and so on."""
    T, K = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for j in range(K):
        back = K - 1 - j
        if back < T:
            y[back:] += taps[:, j].to(x.dtype) * x[:T - back]
    return y


def window_mask(T, size, keep):
    """[T, T]: row i sees the size positions that end with its own, and the first ``keep`` of the sequence up to its own."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep))


def mixed_scores(q, k, scale, cap, talk):
    """q [T, H, D], k [S, G, D] -> [H, T, S]: capped dot products, then every head a combination of all of them."""
    H, G = q.shape[1], k.shape[1]
    raw = torch.stack([soft_cap(q[:, h] @ k[:, h * G // H].t() * scale, cap) for h in range(H)])
    out = torch.zeros_like(raw)
    for h in range(H):
        for g in range(H):
            out[h] += talk[h, g] * raw[g]
    return out


def softmax_with_sink(scores, visible, sink):
    """Softmax over the visible keys whose denominator also holds exp(sink)."""
    s = scores.masked_fill(~visible, -math.inf)
    m = torch.maximum(s.max(-1, keepdim=True).values, sink)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - m))


def talking_attention(q, k, v, scale, cap, talk, sink, size, keep):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]."""
    T, H = q.shape[:2]
    G = k.shape[1]
    scores, seen = mixed_scores(q, k, scale, cap, talk), window_mask(T, size, keep)
    return torch.stack([softmax_with_sink(scores[h], seen, sink[h]) @ v[:, h * G // H] for h in range(H)], 1)


def attention(p, mix, w, h, eps):
    T, H, G, D, V = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    t = lambda n: w[p + n].to(h.dtype)                                                  # noqa: E731
    q = unit_rms(h @ t("q").t(), eps) * t("q.norm")
    k = unit_rms(h @ t("k").t(), eps) * t("k.norm")
    v = h @ t("v").t()
    o = talking_attention(q.view(T, H, D), k.view(T, G, D), v.view(T, G, V), mix["scale"], mix["softcap"], t("talk"), t("sink"),
                          mix["mask"]["size"], mix["mask"]["keep_first"])
    return o.reshape(T, H * V) @ t("o").t()


def dense(p, w, h):
    a = w[p + "act"].to(h.dtype)
    return xielu(h @ w[p + "up"].to(h.dtype).t(), a[0], a[1]) @ w[p + "down"].to(h.dtype).t()


def gated(p, w, h):
    t = lambda n: w[p + n].to(h.dtype)                                                  # noqa: E731
    return (silu(h @ t("gate").t()) * (h @ t("up").t())) @ t("down").t()


def routing(logits, top):
    """The largest logits and a softmax over them alone: (experts [T, top], weights [T, top])."""
    best, idx = torch.sort(logits, -1, descending=True)
    best, idx = best[:, :top], idx[:, :top]
    e = torch.exp(best - best[:, :1])
    return idx, e / e.sum(-1, keepdim=True)


def experts(p, mlp, w, h, gaps=None):
    z = h @ w[p + "router"].to(h.dtype).t() + w[p + "router.b"].to(h.dtype)
    if gaps is not None and mlp["router"]["top"] < mlp["router"]["experts"]:
        best = torch.sort(z, -1, descending=True).values
        gaps.append((best[:, mlp["router"]["top"] - 1] - best[:, mlp["router"]["top"]]) / z.std())
    idx, weight = routing(z, mlp["router"]["top"])
    out = gated(p + "shared.", w, h) if mlp.get("shared") else torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, s = (idx == e).nonzero(as_tuple=True)
        if len(t):
            out[t] += weight[t, s, None] * gated(f"{p}e{e}.", w, h[t])
    return out


def layer(i, spec, cfg, w, x, gaps=None):
    p, eps = f"l{i}.", cfg["norm"]["eps"]
    h = x + causal_conv(x, w[p + "canon1"])
    x = x + norm_plus_one(attention(p + "mix.", spec["mixer"], w, h, eps), w[p + "norm1"], eps) * w[p + "ls1"].to(x.dtype)
    mlp = spec.get("mlp")
    if mlp is not None:
        y = dense(p + "mlp.", w, x) if mlp["kind"] == "dense" else experts(p + "mlp.", mlp, w, x, gaps)
        x = x + norm_plus_one(y, w[p + "norm2"], eps) * w[p + "ls2"].to(x.dtype)
    return x


def forward(cfg, w, tokens, dtype=torch.float64, return_layers=False, gaps=None):
    """Logits [T, vocab] of one sequence (and the stream behind every layer). ``gaps`` collects, per routed layer, how far the last chosen
    expert's logit is ahead of the next one's, over the logits' standard deviation."""
    table = w["embed"].to(dtype)
    x = table[torch.as_tensor(tokens)] + position_vectors(torch.arange(len(tokens)), cfg["width"], dtype)
    layers = []
    for i, spec in enumerate(cfg["layers"]):
        x = layer(i, spec, cfg, w, x, gaps)
        layers.append(x)
    logits = norm_plus_one(x, w["final.norm"], cfg["norm"]["eps"]) @ table.t()
    return (logits, torch.stack(layers)) if return_layers else logits


# ---------------------------------------------------------------------------------------------- small random models
def attention_layer(heads, kv_heads, dim, vdim, size, keep, mlp, scale=0.15, cap=20.0):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": cap,
                                                       "mask": {"size": size, "keep_first": keep}}}


def dense_ff(ff):
    return {"kind": "dense", "ff": ff}


def expert_ff(n, top, ff, shared=0):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": n, "top": top}}
    return dict(m, shared={"ff": shared}) if shared else m


def config(width, vocab, layers, taps=3, eps=1e-5):
    return {"architecture": "Gulazen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps}, "layers": layers}


def weights(cfg, seed=0):
    """Random weights that keep every mechanism visible: unequal norms and layer scales, strong head mixing, sinks of the size of the
    scores, router biases that matter."""
    g = torch.Generator().manual_seed(seed)
    W, out = cfg["width"], {}

    def put(name, *shape, std=1.0, mean=0.0):
        out[name] = (torch.randn(*shape, generator=g) * std + mean).to(torch.bfloat16)

    def mat(name, n, k, gain=1.0):
        put(name, n, k, std=gain * k ** -0.5)

    put("embed", cfg["vocab"], W)
    put("final.norm", W, std=0.2)
    for i, spec in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", spec["mixer"], spec.get("mlp")
        H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        put(p + "canon1", W, cfg["canon"]["taps"], std=0.5)
        for n in "12" if mlp else "1":
            put(f"{p}norm{n}", W, std=0.2)
            put(f"{p}ls{n}", W, std=0.2, mean=0.7)
        q = p + "mix."
        mat(q + "q", H * D, W)
        mat(q + "k", G * D, W)
        mat(q + "v", G * V, W)
        mat(q + "o", W, H * V)
        put(q + "q.norm", H * D, std=0.2, mean=1.0)
        put(q + "k.norm", G * D, std=0.2, mean=1.0)
        out[q + "talk"] = (torch.eye(H) + torch.randn(H, H, generator=g) * 0.5 * H ** -0.5).to(torch.bfloat16)
        put(q + "sink", H, std=1.0, mean=1.0)
        q = p + "mlp."
        if mlp and mlp["kind"] == "dense":
            mat(q + "up", mlp["ff"], W)
            mat(q + "down", W, mlp["ff"])
            put(q + "act", 2, std=0.7)
        elif mlp:
            r, f = mlp["router"], mlp["expert"]["ff"]
            mat(q + "router", r["experts"], W, gain=2.0)
            put(q + "router.b", r["experts"], std=0.5)
            for e in [f"e{e}" for e in range(r["experts"])] + (["shared"] if mlp.get("shared") else []):
                n = mlp["shared"]["ff"] if e == "shared" else f
                mat(f"{q}{e}.gate", n, W, gain=1.5)
                mat(f"{q}{e}.up", n, W, gain=1.5)
                mat(f"{q}{e}.down", W, n)
    return out


def errors(got, want):
    """Per row: root mean square difference of the centred logits over the scale of the expected ones."""
    got, want = got.double().cpu(), want.double()
    got, want = got - got.mean(-1, keepdim=True), want - want.mean(-1, keepdim=True)
    return (got - want).square().mean(-1).sqrt() / want.square().mean().sqrt()


def error(got, want):
    return float(errors(got, want).max())


def decided(cfg, w, tokens, gap=0.03):
    """Rows in which rounding cannot change which experts are chosen."""
    gaps = []
    forward(cfg, w, tokens, torch.float32, gaps=gaps)
    return torch.stack(gaps).min(0).values > gap if gaps else torch.ones(len(tokens), dtype=torch.bool)
