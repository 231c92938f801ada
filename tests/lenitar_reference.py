"""Plain whole-sequence restatement of the Lenitar decoder: one function per mechanism, token by token where the mechanism is a
recurrence, dense masked scores where it is attention, expert by expert where it is routed. The oracle of the Lenitar tests;
it shares nothing with the package. ``cfg`` is the parsed config.json, ``w`` maps tensor names to tensors; everything runs in
``dtype``."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, weight, bias, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight.to(x.dtype) + bias.to(x.dtype)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def lin(w, name, h):
    y = h @ w[name].to(h.dtype).t()
    return y + w[name + ".b"].to(h.dtype) if name + ".b" in w else y


def rotate(x, positions, base, dims):
    """x [T, heads, D]: the first ``dims`` entries are turned pairwise (i, i + dims / 2) by position * base^(-2 i / dims)."""
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    a = (positions.to(torch.float64)[:, None] * f[None, :]).to(x.dtype)[:, None, :]
    u, v, rest = x[..., :half], x[..., half:dims], x[..., dims:]
    return torch.cat((u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a), rest), -1)


def window_mask(T, size):
    """[T, T]: row i sees itself and the size - 1 positions before it."""
    gap = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (gap >= 0) & (gap < size)


def latent_queries(p, mix, w, h, eps):
    """(unrotated [T, H, dim], rotated [T, H, rot]) parts of the queries."""
    T = h.shape[0]
    cq = rms(lin(w, p + "dq", h), eps) * w[p + "dq.norm"].to(h.dtype)
    q = lin(w, p + "uq", cq).view(T, mix["heads"], mix["dim"] + mix["rot_dim"])
    return q[..., :mix["dim"]], rotate(q[..., mix["dim"]:], torch.arange(T), mix["rot"]["base"], mix["rot"]["dims"])


def latent_context(p, mix, w, h, eps):
    """(latent [T, kv_rank], rotated key part [T, rot] shared by all heads)."""
    T, R = h.shape[0], mix["kv_rank"]
    d = lin(w, p + "dkv", h)
    c = rms(d[:, :R], eps) * w[p + "dkv.norm"].to(h.dtype)
    return c, rotate(d[:, None, R:], torch.arange(T), mix["rot"]["base"], mix["rot"]["dims"])[:, 0]


def attention_weights(scores, visible, sink):
    """Softmax over the visible keys whose denominator also holds exp(sink)."""
    s = scores.masked_fill(~visible, -math.inf)
    m = torch.maximum(s.max(-1, keepdim=True).values, sink)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - m))


def latent_heads(qn, qr, c, kr, uk, uv, sink, scale, visible):
    """Per-head attention over the expanded latent: qn [T, H, dim], qr [T, H, rot], c [T, R], kr [T, rot], uk [H, dim, R],
    uv [H, vdim, R] -> [T, H, vdim]."""
    out = []
    for h in range(qn.shape[1]):
        k, v = c @ uk[h].t(), c @ uv[h].t()
        a = attention_weights((qn[:, h] @ k.t() + qr[:, h] @ kr.t()) * scale, visible, sink[h])
        out.append(a @ v)
    return torch.stack(out, 1)


def latent_attention(p, mix, w, h, eps):
    T, H = h.shape[0], mix["heads"]
    qn, qr = latent_queries(p, mix, w, h, eps)
    c, kr = latent_context(p, mix, w, h, eps)
    uk = w[p + "uk"].to(h.dtype).view(H, mix["dim"], mix["kv_rank"])
    uv = w[p + "uv"].to(h.dtype).view(H, mix["vdim"], mix["kv_rank"])
    o = latent_heads(qn, qr, c, kr, uk, uv, w[p + "sink"].to(h.dtype), mix["scale"], window_mask(T, mix["mask"]["size"]))
    return lin(w, p + "o", o.reshape(T, -1) * sigmoid(lin(w, p + "g", h)))


def soft_cap(x, cap):
    return cap * torch.tanh(x / cap)


def mlstm_scan(q, k, v, i, f, state):
    """q, k [T, H, D], v [T, H, V], log gates i, f [T, H]; state (S [H, D, V], n [H, D], m [H]) -> (o [T, H, V], state)."""
    S, n, m = state
    out = []
    for t in range(q.shape[0]):
        new = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - new)[:, None], torch.exp(i[t] - new)[:, None]
        S = keep[..., None] * S + (take * k[t])[:, :, None] * v[t][:, None, :]
        n = keep * n + take * k[t]
        m = new
        size = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append((S * q[t][:, :, None]).sum(1) / size[:, None])
    return torch.stack(out), (S, n, m)


def mlstm_start(H, D, V, dtype=torch.float64):
    return torch.zeros(H, D, V, dtype=dtype), torch.zeros(H, D, dtype=dtype), torch.zeros(H, dtype=dtype)


def mlstm_gates(zi, zf, cap):
    """Log input gate and log forget gate of the projections."""
    return soft_cap(zi, cap), torch.nn.functional.logsigmoid(soft_cap(zf, cap))


def mlstm(p, mix, w, h, eps):
    T, H, D, V = h.shape[0], mix["heads"], mix["dim"], mix["vdim"]
    q = (lin(w, p + "q", h) * D ** -0.5).view(T, H, D)
    k, v = lin(w, p + "k", h).view(T, H, D), lin(w, p + "v", h).view(T, H, V)
    i, f = mlstm_gates(lin(w, p + "i", h), lin(w, p + "f", h), mix["gate_cap"])
    o, _ = mlstm_scan(q, k, v, i, f, mlstm_start(H, D, V, h.dtype))
    o = rms(o, eps).reshape(T, H * V) * w[p + "norm"].to(h.dtype)
    return lin(w, p + "o", o * sigmoid(lin(w, p + "g", h)))


def route(z, top, groups, keep):
    """Router logits of one token -> [(expert, weight)]: the best experts of the best groups, weighted by their scores."""
    s = sigmoid(z)
    E = s.numel()
    size = E // groups
    value = [sum(sorted(s[g * size:(g + 1) * size].tolist(), reverse=True)[:2]) for g in range(groups)]
    best = sorted(range(groups), key=lambda g: (-value[g], g))[:keep]
    allowed = [e for e in range(E) if e // size in best]
    return [(e, s[e]) for e in sorted(allowed, key=lambda e: (-float(s[e]), e))[:top]]


def expert(p, w, h):
    g = lin(w, p + "gate", h)
    return lin(w, p + "down", g * sigmoid(g) * lin(w, p + "up", h))


def mixture(p, mlp, w, h):
    r = mlp["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    z = lin(w, p + "router", h)
    out = []
    for t in range(h.shape[0]):
        y = torch.zeros_like(h[t])
        for e, s in route(z[t], r["top"], g["count"], g["keep"]):
            y = y + s * expert(f"{p}e{e}.", w, h[t])
        out.append(y)
    return torch.stack(out)


def forward(cfg, w, tokens, dtype=torch.float64, return_layers=False):
    """Logits of every position [T, vocab] (and the residual stream behind every layer)."""
    eps = cfg["norm"]["eps"]
    x = w["embed"].to(dtype)[torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    layers = []
    for i, layer in enumerate(cfg["layers"]):
        h = layer_norm(x, w[f"l{i}.norm1"], w[f"l{i}.norm1.b"], eps)
        mixer = {"latent_attention": latent_attention, "mlstm": mlstm}[layer["type"]]
        y = mixer(f"l{i}.mix.", layer["mixer"], w, h, eps)
        if layer.get("mlp"):
            y = y + mixture(f"l{i}.mlp.", layer["mlp"], w, h)
        x = x + y
        layers.append(x)
    logits = layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].to(dtype).t()
    return (logits, layers) if return_layers else logits


# ---------------------------------------------------------------------------------------------- models for the tests
def moe(experts, top, ff, groups=1, keep=1):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}, "expert": {"ff": ff}}


def latent(heads, dim, rot, vdim, kv_rank, q_rank, window, mlp=None, base=10000.0, scale=0.2):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "mask": {"size": window},
         "rot": {"dims": rot, "base": base}, "scale": scale}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def mlstm_layer(heads, dim, vdim, cap, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def config(width, vocab, layers, eps=1e-5, scale=1.0):
    return {"architecture": "Lenitar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}


def weights(cfg, seed=0, gain=1.0):
    """bf16-valued random weights that keep every path of the model loud: unit-variance projections, norms around one, gates
    from closed to open, sinks that matter."""
    g = torch.Generator().manual_seed(seed)
    W, w = cfg["width"], {}

    def mat(name, rows, cols, s=1.0):
        w[name] = torch.randn(rows, cols, generator=g) * (s * gain / math.sqrt(cols))

    def vec(name, n, s=0.3, mean=0.0):
        w[name] = torch.randn(n, generator=g) * s + mean

    w["embed"] = torch.randn(cfg["vocab"], W, generator=g) / cfg["embedding"]["scale"]
    mat("head", cfg["vocab"], W)
    vec("final.norm", W, 0.3, 1.0)
    vec("final.norm.b", W)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        vec(f"l{i}.norm1", W, 0.3, 1.0)
        vec(f"l{i}.norm1.b", W)
        if layer["type"] == "mlstm":
            qk, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, rows in (("q", qk), ("k", qk), ("v", v), ("g", v)):
                mat(p + n, rows, W)
            for n, mean in (("i", -1.0), ("f", 3.0)):
                mat(p + n, m["heads"], W)
                vec(p + n + ".b", m["heads"], 1.5, mean)
            vec(p + "norm", v, 0.3, 1.0)
            mat(p + "o", W, v)
        else:
            H, R = m["heads"], m["kv_rank"]
            mat(p + "dq", m["q_rank"], W)
            vec(p + "dq.norm", m["q_rank"], 0.3, 1.0)
            mat(p + "uq", H * (m["dim"] + m["rot_dim"]), m["q_rank"])
            mat(p + "dkv", R + m["rot_dim"], W)
            vec(p + "dkv.norm", R, 0.3, 1.0)
            mat(p + "uk", H * m["dim"], R)
            mat(p + "uv", H * m["vdim"], R)
            vec(p + "sink", H, 1.0, 1.0)
            mat(p + "g", H * m["vdim"], W)
            mat(p + "o", W, H * m["vdim"])
        if layer["mlp"]:
            q, ff = f"l{i}.mlp.", layer["mlp"]["expert"]["ff"]
            mat(q + "router", layer["mlp"]["router"]["experts"], W, 2.0)
            for e in range(layer["mlp"]["router"]["experts"]):
                mat(f"{q}e{e}.gate", ff, W)
                mat(f"{q}e{e}.up", ff, W)
                mat(f"{q}e{e}.down", W, ff)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


def error(got, want):
    """Largest over the rows: root mean square difference of the logits (mean removed), relative to the logits' own."""
    return float(errors(got, want).max())


def errors(got, want):
    got, want = got.double().cpu(), want.double()
    d = got - want
    d, c = d - d.mean(-1, keepdim=True), want - want.mean(-1, keepdim=True)
    return d.square().mean(-1).sqrt() / c.square().mean().sqrt()
