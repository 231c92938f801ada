"""Plain whole-sequence restatement of the Kasuvik decoder: one function per mechanism, token by token where the mechanism is a
recurrence, dense masked scores where it is attention. The oracle of the Kasuvik tests; it shares nothing with the package.
``cfg`` is the parsed config.json, ``w`` maps tensor names to tensors; everything runs in ``dtype``."""
import math

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight.to(x.dtype)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def lin(w, name, h):
    y = h @ w[name].to(h.dtype).t()
    return y + w[name + ".b"].to(h.dtype) if name + ".b" in w else y


def causal_conv(u, taps):
    """u [T, C], taps [C, n]: y_t = sum_j taps[:, j] u_(t - n + 1 + j), zeros before the start."""
    n = taps.shape[1]
    padded = torch.cat((torch.zeros(n - 1, u.shape[1], dtype=u.dtype), u))
    return sum(taps[:, j].to(u.dtype) * padded[j:j + u.shape[0]] for j in range(n))


def rotate(x, positions, base, dims):
    """x [T, heads, D]: neighbouring entries (2 i, 2 i + 1) of the first ``dims`` are turned by position * base^(-2 i / dims)."""
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    a = (positions.to(torch.float64)[:, None] * f[None, :]).to(x.dtype)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    turned = torch.stack((u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a)), -1).flatten(-2)
    return torch.cat((turned, x[..., dims:]), -1)


def pooled(x, pool):
    """x [T, ...] -> the means of its whole blocks of ``pool`` rows."""
    n = x.shape[0] // pool
    return x[:n * pool].reshape(n, pool, *x.shape[1:]).mean(1)


def visible_tokens(T, size):
    """[T, T]: row i sees itself and the size - 1 positions before it."""
    gap = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (gap >= 0) & (gap < size)


def visible_blocks(T, size, pool):
    """[T, T // pool]: row i sees the blocks that end at i - size or before."""
    last = torch.arange(T // pool) * pool + pool - 1
    return last[None, :] <= torch.arange(T)[:, None] - size


def pooled_attention(q, k, v, scale, size, pool):
    """q [T, H, D], k [T, G, D], v [T, G, V] as the cache holds them -> [T, H, V]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    kk, vv = torch.cat((k, pooled(k, pool))), torch.cat((v, pooled(v, pool)))
    seen = torch.cat((visible_tokens(T, size), visible_blocks(T, size, pool)), 1)
    out = []
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ kk[:, g].t()) * scale).masked_fill(~seen, -math.inf)
        out.append(torch.softmax(s, -1) @ vv[:, g])
    return torch.stack(out, 1)


def attention_inputs(p, m, w, h):
    """Queries (times the head's temperature), keys and values after convolution and rotation."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = (causal_conv(lin(w, p + n, h), w[p + n + ".conv"]) for n in "qkv")
    pos = torch.arange(T)
    rot = lambda t: rotate(t, pos, m["rot"]["base"], m["rot"]["dims"])                  # noqa: E731
    q = rot(q.view(T, H, m["dim"])) * w[p + "temp"].to(h.dtype)[None, :, None]
    return q, rot(k.view(T, G, m["dim"])), v.view(T, G, m["vdim"])


def attention(p, m, w, h):
    q, k, v = attention_inputs(p, m, w, h)
    o = pooled_attention(q, k, v, m["scale"], m["mask"]["size"], m["mask"]["pool"])
    return lin(w, p + "o", o.reshape(h.shape[0], -1))


def selective_scan(x, dt, B, C, A, D, S):
    """x, dt [T, c], B, C [T, n], A [c, n], D [c], state S [c, n] -> (y [T, c], S)."""
    out = []
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        out.append((S * C[t][None, :]).sum(-1) + D * x[t])
    return torch.stack(out), S


def mamba(p, m, w, h):
    inner, n, r = m["inner"], m["state"], m["dt_rank"]
    xz = lin(w, p + "in", h)
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(causal_conv(x, w[p + "conv"]) + w[p + "conv.b"].to(h.dtype))
    d = lin(w, p + "x", x)
    dt = softplus(lin(w, p + "dt", d[:, :r]))
    A = -torch.exp(w[p + "A_log"].to(h.dtype))
    y, _ = selective_scan(x, dt, d[:, r:r + n], d[:, r + n:], A, w[p + "D"].to(h.dtype), torch.zeros(inner, n, dtype=h.dtype))
    return lin(w, p + "o", y * silu(z))


def parallel(p, m, w, h, eps):
    left = rms_norm(attention(p + "left.", m["left"], w, h), w[p + "left.out"], eps)
    right = rms_norm(mamba(p + "right.", m["right"], w, h), w[p + "right.out"], eps)
    return (left + right) / 2


def delta_scan(r, k, v, decay, rate, S):
    """r, k, decay, rate [T, H, D], v [T, H, V], state S [H, D, V] -> (o [T, H, V], S)."""
    u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    out = []
    for t in range(r.shape[0]):
        recalled = torch.einsum("hd,hdv->hv", u[t], S)
        S = decay[t][..., None] * S - (rate[t] * u[t])[..., None] * recalled[:, None, :] + k[t][..., None] * v[t][:, None, :]
        out.append(torch.einsum("hd,hdv->hv", r[t], S))
    return torch.stack(out), S


def delta_decay(p, w, h):
    z = lin(w, p + "w2", torch.tanh(lin(w, p + "w1", h))) + w[p + "w0"].to(h.dtype)
    return torch.exp(-math.exp(-0.5) * sigmoid(z))


def general_delta(p, m, w, h, eps):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    r, k, v = (lin(w, p + n, h).view(T, H, D) for n in "rkv")
    o, _ = delta_scan(r, k, v, delta_decay(p, w, h).view(T, H, D), sigmoid(lin(w, p + "a", h)).view(T, H, D), torch.zeros(H, D, D, dtype=h.dtype))
    o = unit_rms(o, eps).reshape(T, H * D) * w[p + "norm"].to(h.dtype)
    return lin(w, p + "o", o * sigmoid(lin(w, p + "g", h)))


def feed_forward(p, w, h):
    return lin(w, p + "down", torch.relu(lin(w, p + "gate", h)) * lin(w, p + "up", h))


def forward(cfg, w, tokens, dtype=torch.float64, return_layers=False):
    """Logits of every position [T, vocab] (and the residual stream behind every layer)."""
    eps = cfg["norm"]["eps"]
    x = w["embed"].to(dtype)[torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    layers = []
    for i, layer in enumerate(cfg["layers"]):
        h = rms_norm(x, w[f"l{i}.norm1"], eps)
        y = {"parallel": parallel, "general_delta": general_delta}[layer["type"]](f"l{i}.mix.", layer["mixer"], w, h, eps)
        x = x + rms_norm(y, w[f"l{i}.norm1b"], eps)
        if layer.get("mlp"):
            y = feed_forward(f"l{i}.mlp.", w, rms_norm(x, w[f"l{i}.norm2"], eps))
            x = x + rms_norm(y, w[f"l{i}.norm2b"], eps)
        layers.append(x)
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].to(dtype).t()
    return (logits, layers) if return_layers else logits


# ---------------------------------------------------------------------------------------------- models for the tests
def parallel_layer(heads, kv_heads, dim, vdim, window, pool, inner, state, dt_rank, ff=0, conv=3, mamba_conv=4, rot=None, base=10000.0,
                   scale=0.2):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "mask": {"size": window, "pool": pool},
            "rot": {"dims": dim if rot is None else rot, "base": base}, "scale": scale}
    right = {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": mamba_conv}
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def delta_layer(heads, dim, ff=0):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width, vocab, layers, eps=1e-5, scale=1.0):
    return {"architecture": "Kasuvik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}


def weights(cfg, seed=0, rank=12):
    """bf16-valued random weights that keep every path of the model loud: unit-variance projections, norms around one, removal
    and decay rates from small to large, step sizes and state decays over a wide range, temperatures that sharpen. ``rank``: of the
    delta rule's decay projection."""
    g = torch.Generator().manual_seed(seed)
    W, w = cfg["width"], {}

    def mat(name, rows, cols, s=1.0):
        w[name] = torch.randn(rows, cols, generator=g) * (s / math.sqrt(cols))

    def vec(name, n, s=0.3, mean=0.0):
        w[name] = torch.randn(n, generator=g) * s + mean

    w["embed"] = torch.randn(cfg["vocab"], W, generator=g) / cfg["embedding"]["scale"]
    mat("head", cfg["vocab"], W)
    vec("final.norm", W, 0.3, 1.0)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if layer["mlp"] else ()):
            vec(f"l{i}.{n}", W, 0.3, 1.0)
        if layer["type"] == "general_delta":
            n = m["heads"] * m["dim"]
            for t in "rkvg":
                mat(p + t, n, W)
            mat(p + "a", n, W, 1.5)
            vec(p + "a.b", n, 1.0)
            mat(p + "w1", rank, W)
            mat(p + "w2", n, rank, 2.0)
            vec(p + "w0", n, 2.0, -2.0)
            vec(p + "norm", n, 0.3, 1.0)
            mat(p + "o", W, n)
        else:
            a, b, l, r = m["left"], m["right"], p + "left.", p + "right."
            q, k, v = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"]
            for t, rows in (("q", q), ("k", k), ("v", v)):
                mat(l + t, rows, W)
                vec(l + t + ".b", rows)
                w[l + t + ".conv"] = torch.randn(rows, a["conv"], generator=g) / math.sqrt(a["conv"])
            vec(l + "temp", a["heads"], 0.5, 1.5)
            mat(l + "o", W, a["heads"] * a["vdim"])
            c, n = b["inner"], b["state"]
            mat(r + "in", 2 * c, W)
            w[r + "conv"] = torch.randn(c, b["conv"], generator=g) / math.sqrt(b["conv"])
            vec(r + "conv.b", c)
            mat(r + "x", b["dt_rank"] + 2 * n, c, 2.0)
            mat(r + "dt", c, b["dt_rank"])
            vec(r + "dt.b", c, 1.5, -3.0)
            w[r + "A_log"] = torch.randn(c, n, generator=g) * 1.2
            vec(r + "D", c, 0.5, 1.0)
            mat(r + "o", W, c)
            vec(l + "out", W, 0.3, 1.0)
            vec(r + "out", W, 0.3, 1.0)
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            mat(f"l{i}.mlp.gate", ff, W)
            mat(f"l{i}.mlp.up", ff, W)
            mat(f"l{i}.mlp.down", W, ff)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


def error(got, want):
    """Largest over the rows: root mean square difference of the logits (mean removed), relative to the logits' own."""
    return float(errors(got, want).max())


def errors(got, want):
    got, want = got.double().cpu(), want.double()
    d = got - want
    d, c = d - d.mean(-1, keepdim=True), want - want.mean(-1, keepdim=True)
    return d.square().mean(-1).sqrt() / c.square().mean().sqrt()
