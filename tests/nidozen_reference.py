"""Plain whole-sequence restatement of the Nidozen decoder: one function per mechanism, token by token where the mechanism
is a recurrence, dense masked scores where it is attention. The oracle of the Nidozen tests; it shares nothing with the
package. ``cfg`` is the parsed config.json, ``w`` maps tensor names to tensors; everything runs in ``dtype``."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


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


def chunk_mask(T, size):
    i = torch.arange(T)
    return (i[None, :] <= i[:, None]) & (i[None, :] // size == i[:, None] // size)


def attention_heads(q, k, v, scale, visible):
    """q [T, H, D], k [T, G, D], v [T, G, V]; ``visible`` [T, T] bool."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].t()) * scale
        s = s.masked_fill(~visible, -math.inf)
        out.append(torch.softmax(s, -1) @ v[:, g])
    return torch.stack(out, 1)


def attention_keys_values(p, mix, w, h, eps):
    T = h.shape[0]
    G = mix["kv_heads"]
    k = rms(lin(w, p + "k", h), eps) * w[p + "k.norm"].to(h.dtype)
    k = rotate(k.view(T, G, mix["dim"]), torch.arange(T), mix["rot"]["base"], mix["rot"]["dims"])
    v = rms(lin(w, p + "v", h).view(T, G, mix["vdim"]), eps)
    return k, v


def attention(p, mix, w, h, eps, shared):
    T = h.shape[0]
    q = rms(lin(w, p + "q", h), eps) * w[p + "q.norm"].to(h.dtype)
    q = rotate(q.view(T, mix["heads"], mix["dim"]), torch.arange(T), mix["rot"]["base"], mix["rot"]["dims"])
    k, v = shared if shared is not None else attention_keys_values(p, mix, w, h, eps)
    o = attention_heads(q, k, v, mix["scale"], chunk_mask(T, mix["mask"]["size"]))
    return lin(w, p + "o", o.reshape(T, -1)), (k, v)


def mingru(p, mix, w, h, state=None):
    z = torch.sigmoid(lin(w, p + "z", h))
    u = lin(w, p + "x", h)
    cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    S = torch.zeros_like(z[0]) if state is None else state
    rows = []
    for t in range(h.shape[0]):
        S = (1 - z[t]) * S + z[t] * cand[t]
        rows.append(S)
    g = lin(w, p + "g", h)
    return lin(w, p + "o", torch.stack(rows) * (g * torch.sigmoid(g)))


def gla_scan(q, k, v, alpha, S):
    """q, k, alpha [T, H, D], v [T, H, V], S [H, D, V]: S <- diag(alpha) S + k v^T, o = S^T q."""
    out = []
    for t in range(q.shape[0]):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def gla(p, mix, w, h, eps):
    T, H, D, V = h.shape[0], mix["heads"], mix["dim"], mix["vdim"]
    q = (lin(w, p + "q", h) * D ** -0.5).view(T, H, D)
    k = lin(w, p + "k", h).view(T, H, D)
    v = lin(w, p + "v", h).view(T, H, V)
    z = lin(w, p + "a2", lin(w, p + "a1", h)).view(T, H, D)
    alpha = torch.sigmoid(z) ** (1.0 / mix["tau"])
    o, _ = gla_scan(q, k, v, alpha, torch.zeros(H, D, V, dtype=h.dtype))
    o = (rms(o, eps) * w[p + "norm"].to(h.dtype)).reshape(T, H * V)
    g = lin(w, p + "g", h)
    return lin(w, p + "o", o * (g * torch.sigmoid(g)))


def dense_relu2(p, w, h):
    a = torch.relu(lin(w, p + "up", h))
    return lin(w, p + "down", a * a)


def forward(cfg, w, tokens, dtype=torch.float64, return_layers=False):
    """Logits of every position [T, vocab] (and the residual stream behind every layer)."""
    eps = cfg["norm"]["eps"]
    x = w["embed"].to(dtype)[torch.as_tensor(tokens)]
    kept, layers = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, mix = f"l{i}.mix.", layer["mixer"]
        if layer["type"] == "mingru":
            y = mingru(p, mix, w, x)
        elif layer["type"] == "gla":
            y = gla(p, mix, w, x, eps)
        else:
            y, kept[i] = attention(p, mix, w, x, eps, kept[mix["kv_from"]] if mix.get("kv_from") is not None else None)
        x = x + rms(y, eps) * w[f"l{i}.norm1"].to(dtype)
        if layer.get("mlp"):
            assert layer["mlp"]["kind"] == "dense"
            x = x + rms(dense_relu2(f"l{i}.mlp.", w, x), eps) * w[f"l{i}.norm2"].to(dtype)
        layers.append(x)
    logits = (rms(x, eps) * w["final.norm"].to(dtype)) @ w["head"].to(dtype).t()
    return (logits, layers) if return_layers else logits


def greedy(cfg, w, prompt, n, dtype=torch.float64):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(forward(cfg, w, ids, dtype)[-1].argmax()))
    return ids[len(prompt):]


# ---------------------------------------------------------------------------------------------- models for the tests
def attn(heads, kv, dim, vdim, chunk, rot, base=10000.0, scale=0.25, ff=0, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "rot": {"dims": rot, "base": base},
         "scale": scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def gla_layer(heads, dim, vdim, tau, ff=0):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def mingru_layer(width, ff=0):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Nidozen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


def weights(cfg, seed=0, rank=8, gain=1.0):
    """bf16-valued random weights that keep every path of the model loud: unit-variance projections, norms around one,
    decays from almost none to strong."""
    g = torch.Generator().manual_seed(seed)
    W, w = cfg["width"], {}

    def mat(name, rows, cols, s=1.0):
        w[name] = torch.randn(rows, cols, generator=g) * (s * gain / math.sqrt(cols))

    def vec(name, n, s=0.5, mean=0.0):
        w[name] = torch.randn(n, generator=g) * s + mean

    def number(name):
        w[name] = torch.rand((), generator=g) + 0.5

    w["embed"] = torch.randn(cfg["vocab"], W, generator=g)
    mat("head", cfg["vocab"], W)
    number("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        number(f"l{i}.norm1")
        if layer["type"] == "mingru":
            for n in "zxg":
                mat(p + n, m["width"], W)
            vec(p + "z.b", m["width"], 1.0, -1.5)        # slow and fast channels
            vec(p + "x.b", m["width"])
            mat(p + "o", W, m["width"])
        elif layer["type"] == "gla":
            qk, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, rows in (("q", qk), ("k", qk), ("v", v), ("g", v)):
                mat(p + n, rows, W)
            mat(p + "a1", rank, W)
            mat(p + "a2", qk, rank)
            vec(p + "a2.b", qk, 2.0, 2.0)
            vec(p + "norm", m["vdim"], 0.3, 1.0)
            mat(p + "o", W, v)
        else:
            q, k, v = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
            mat(p + "q", q, W)
            vec(p + "q.b", q)
            vec(p + "q.norm", q, 0.3, 1.0)
            if m.get("kv_from") is None:
                mat(p + "k", k, W)
                vec(p + "k.b", k)
                vec(p + "k.norm", k, 0.3, 1.0)
                mat(p + "v", v, W)
                vec(p + "v.b", v)
            mat(p + "o", W, m["heads"] * m["vdim"])
            vec(p + "o.b", W)
        if layer["mlp"]:
            number(f"l{i}.norm2")
            mat(f"l{i}.mlp.up", layer["mlp"]["ff"], W)
            mat(f"l{i}.mlp.down", W, layer["mlp"]["ff"])
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


def error(got, want):
    """Largest over the rows: root mean square difference of the logits (mean removed), relative to the logits' own."""
    got, want = got.double().cpu(), want.double()
    d = got - want
    d, c = d - d.mean(-1, keepdim=True), want - want.mean(-1, keepdim=True)
    return float((d.square().mean(-1).sqrt() / c.square().mean().sqrt()).max())
