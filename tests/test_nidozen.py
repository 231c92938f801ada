"""Nidozen: every mechanism alone and whole models against the plain restatement in nidozen_reference.py - prompts, decoding,
portions, unequal batches, reused pages and slots, chunk edges, greedy generation through the engine and the server."""
import json

import pytest
import torch

import nidozen_reference as R
from eredu_b200 import ops
from eredu_b200.models.config import ModelConfig
from eredu_b200.models.llama import ForwardBatch, build_from_tensors
from eredu_b200.ops import SamplingParams
from eredu_b200.runtime.engine import Engine

CASES = [pytest.param("cpu", torch.float32, id="cpu-fp32"), pytest.param("cuda", torch.float32, marks=pytest.mark.gpu, id="gpu-fp32"),
         pytest.param("cuda", torch.bfloat16, marks=pytest.mark.gpu, id="gpu-bf16")]
both = pytest.mark.parametrize("dev,dt", CASES)

# Sizes that are unequal where they can be; grouped and ungrouped heads; chunks that start inside pages and on them; keys read
# by a later layer under another mask and scale; every layer kind with and without a feed-forward.
MIXED = R.config(96, 211, [R.gla_layer(3, 24, 40, 4.0, ff=72), R.attn(6, 2, 40, 24, 37, 8, 1000.0, 0.3),
                           R.attn(6, 2, 40, 24, 20, 8, 1000.0, 0.2, ff=88, kv_from=1), R.mingru_layer(72, ff=40),
                           R.attn(2, 2, 128, 128, 64, 128, 20000.0, 0.1, ff=48), R.attn(4, 1, 16, 72, 50, 2, scale=0.4)], eps=3e-5)
# Sizes the tensor-core kernels do not take (not multiples of 8, values wider than their tiles, odd widths), decays without a root.
ODD = R.config(70, 131, [R.mingru_layer(33), R.attn(3, 1, 20, 12, 9, 6, 500.0, 0.5, ff=51), R.gla_layer(1, 20, 300, 1.0, ff=30),
                         R.attn(2, 1, 136, 200, 48, 136, scale=0.1), R.gla_layer(2, 128, 256, 1.0)])
SMALL = R.config(64, 97, [R.gla_layer(2, 16, 24, 2.0), R.attn(4, 2, 24, 16, 40, 8, ff=48), R.mingru_layer(56)])
LIMIT = {torch.float32: 2e-4, torch.bfloat16: 0.06}


def engine_for(cfg, w, dev, dt, **kw):
    mc = ModelConfig.from_hf_dict(json.loads(json.dumps(cfg)))
    model = build_from_tensors(mc, w.__getitem__, w.__contains__, dev, dt)
    return Engine(model, **{"max_batch": 4, "max_seq_len": 512, **kw})


def prompt(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def feed(eng, seq, tokens, sizes):
    """Tokens in portions of the given sizes (the last one repeated); logits of every position."""
    rows, at, i = [], 0, 0
    while at < len(tokens):
        n = sizes[min(i, len(sizes) - 1)]
        part = tokens[at:at + n]
        rows.append(eng.forward_tokens([(seq, part, range(len(part)))]))
        at, i = at + n, i + 1
    return torch.cat(rows)


# ---------------------------------------------------------------------------------------------- configuration
def test_config_keeps_every_layer_and_round_trips():
    cfg = ModelConfig.from_hf_dict(MIXED)
    assert cfg.model_type == "nidozen" and cfg.num_hidden_layers == 6 and cfg.is_hybrid and cfg.vocab_size == 211
    assert [cfg.layer_has_kv(i) for i in range(6)] == [False, True, False, False, True, True]
    assert cfg.layer_kv_donor(2) == 1 and cfg.layer_kv_dims(4) == (2, 128, 128) and cfg.layer_kv_dims(5) == (1, 16, 72)
    assert cfg.layer_state_shape(0) == (3, 24, 40) and cfg.layer_state_shape(3) == (72,) and cfg.layer_state_shape(1) is None
    assert cfg.mixers[2].chunk == 20 and cfg.mixers[2].scale == 0.2 and cfg.rms_norm_eps == 3e-5
    assert ModelConfig.from_hf_dict(cfg.to_hf_dict()).mixers == cfg.mixers
    wrong = json.loads(json.dumps(MIXED))
    wrong["layers"][2]["mixer"]["kv_from"] = 0
    with pytest.raises(ValueError):
        ModelConfig.from_hf_dict(wrong)
    wrong["layers"][2]["mixer"].update(kv_from=1, kv_heads=3)
    with pytest.raises(ValueError):
        ModelConfig.from_hf_dict(wrong)


def test_cache_pools_layers_by_geometry_and_states_by_layer():
    eng = engine_for(MIXED, R.weights(MIXED), "cpu", torch.float32, state_slots=3)
    assert len(eng.kv.pools) == 3 and eng.kv.layer(1)[0].data_ptr() == eng.kv.layer(2)[0].data_ptr()
    assert eng.kv.layer(1)[0].shape[1:] == (2, 16, 40) and eng.kv.layer(1)[1].shape[1:] == (2, 16, 24)
    assert eng.kv.layer_state[0].shape == (3, 3, 24, 40) and eng.kv.layer_state[3].shape == (3, 72)
    with pytest.raises(NotImplementedError):
        from eredu_b200.runtime.kv_residency import KVHostTier

        KVHostTier(eng)


# ---------------------------------------------------------------------------------------------- mechanisms
def close(got, want, dt, scale=None):
    got, want = got.double().cpu(), want.double()
    s = scale or float(want.abs().max())
    limit = 2e-5 if dt == torch.float32 else 1.2e-2
    assert got.shape == want.shape and float((got - want).abs().max()) <= limit * s, float((got - want).abs().max()) / s


def rand(*shape, seed=0, dt=torch.float32):
    """Random values exact in bf16, on the CPU in fp64."""
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)).to(torch.bfloat16).double()


@both
@pytest.mark.parametrize("width", [33, 96, 1000, 1028, 2500, 9000])
def test_norm_on_the_output_and_fp32_stream(dev, dt, width):
    y, x = rand(5, width, seed=1), rand(5, width, seed=2) * 3 + 1e-3
    x = x.float()
    for w in (torch.tensor([0.7]), torch.rand(width) + 0.5):
        got, act = ops.rms_residual(y.to(dev, dt), w.to(dev), 1e-4, residual=x.to(dev), act_dtype=dt)
        want = x.double() + R.rms(y, 1e-4) * w.double()
        close(got, want, torch.float32)
        close(act, want, dt)
        plain = ops.rms_residual(x.to(dev), w.to(dev), 1e-4, act_dtype=dt)[1]
        close(plain, R.rms(x.double(), 1e-4) * w.double(), dt)
    table = rand(11, width, seed=3)
    ids = torch.tensor([3, 0, 10], dtype=torch.int32)
    s, a = ops.embedding_stream(ids.to(dev), table.to(dev, dt))
    assert torch.equal(s.double().cpu(), table[ids.long()]) and torch.equal(a.double().cpu(), table[ids.long()])


@both
@pytest.mark.parametrize("m,n,k", [(1, 40, 64), (3, 131, 33), (40, 96, 72), (300, 200, 128), (300, 51, 70), (64, 1000, 20)])
def test_linear_with_bias_and_squared_relu(dev, dt, m, n, k):
    x, w, b = rand(m, k, seed=1), rand(n, k, seed=2), rand(n, seed=3)
    y = x @ w.t() + b
    close(ops.linear(x.to(dev, dt), w.to(dev, dt), bias=b.to(dev, dt)), y, dt)
    close(ops.linear(x.to(dev, dt), w.to(dev, dt), bias=b.to(dev, dt), activation="relu2"), torch.relu(y) ** 2, dt)
    close(ops.linear(x.to(dev, dt), w.to(dev, dt), out_dtype=torch.float32, activation="relu2"), torch.relu(x @ w.t()) ** 2, torch.float32
          if dt == torch.float32 else dt)


@both
@pytest.mark.parametrize("nq,nkv,dk,dv,rot", [(6, 2, 40, 24, 8), (2, 2, 128, 64, 128), (3, 1, 20, 12, 6), (4, 4, 16, 200, 0)])
def test_query_key_value_preparation(dev, dt, nq, nkv, dk, dv, rot):
    M, eps = 7, 1e-3
    positions = torch.tensor([0, 1, 15, 16, 17, 1000, 5])
    x = rand(M, (nq + nkv) * dk + nkv * dv, seed=4) * 2
    qw, kw = rand(nq * dk, seed=5) + 1, rand(nkv * dk, seed=6) + 1
    inv = torch.tensor([300.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float32)
    slots = torch.tensor([17, 40, 2 * 16 + 15, 3 * 16, 5, -1, 63])
    kc, vc = torch.zeros(4, nkv, 16, dk, device=dev, dtype=dt), torch.zeros(4, nkv, 16, dv, device=dev, dtype=dt)
    args = (positions.int().to(dev), slots.to(dev), inv.to(dev), kc, vc, nq, nkv, dk, dv, qw.float().to(dev), kw.float().to(dev), eps)
    got = ops.qkv_prepare(x.to(dev, dt), *args, value_norm=True)
    a = (positions.double()[:, None] * inv.double()[None])[:, None, :]

    def turned(t, w, heads):
        t = (R.rms(t, eps) * w).view(M, heads, dk)
        u, v = t[..., :rot // 2], t[..., rot // 2:rot]
        return torch.cat((u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin(), t[..., rot:]), -1)

    q, k = turned(x[:, :nq * dk], qw, nq), turned(x[:, nq * dk:(nq + nkv) * dk], kw, nkv)
    v = R.rms(x[:, (nq + nkv) * dk:].view(M, nkv, dv), eps)
    limit = torch.bfloat16 if dt == torch.bfloat16 else torch.float32
    tol = 5e-4 if limit == torch.float32 else 1.2e-2                  # fp32 angles at position 1000
    assert float((got.double().cpu() - q).abs().max()) <= tol * float(q.abs().max())
    for m, s in enumerate(slots.tolist()):
        if s >= 0:
            assert float((kc[s // 16, :, s % 16].double().cpu() - k[m]).abs().max()) <= tol * float(k.abs().max())
            close(vc[s // 16, :, s % 16], v[m], dt)
    filled = {s for s in slots.tolist() if s >= 0}
    for s in range(64):
        if s not in filled:
            assert not kc[s // 16, :, s % 16].any() and not vc[s // 16, :, s % 16].any()
    before = kc.clone()
    only_q = ops.qkv_prepare(x[:, :nq * dk].contiguous().to(dev, dt), *args, append=False)
    assert torch.equal(only_q, got) and torch.equal(kc, before)


def paged(rows, pages, n_pages, dev, dt):
    """[T, G, D] rows scattered over the given pages of a pool."""
    T, G, D = rows.shape
    pool = torch.full((n_pages, G, 16, D), 7.0, device=dev, dtype=dt)
    for t in range(T):
        pool[pages[t // 16], :, t % 16] = rows[t].to(dev, dt)
    return pool


@both
@pytest.mark.parametrize("H,G,dk,dv,chunk", [(4, 2, 64, 64, 80), (6, 2, 40, 24, 37), (4, 4, 128, 64, 16), (2, 1, 48, 128, 100), (8, 1, 128, 128, 200),
                                             (3, 1, 20, 12, 9), (2, 1, 136, 200, 48), (4, 1, 16, 72, 1), (4, 2, 64, 64, 0)])
def test_chunked_attention_sees_its_chunk_and_nothing_else(dev, dt, H, G, dk, dv, chunk):
    """Keys at chunk edges are made to stand out: one just inside or outside a query's chunk decides the whole row."""
    T = 330
    q, k, v = rand(T, H, dk, seed=1), rand(T, G, dk, seed=2) * 0.2, rand(T, G, dv, seed=3)
    size = chunk or 10 ** 6
    edges = [p for c in range(0, T, size) for p in (c - 1, c, c + 1) if 0 <= p < T] + [150, 15, 16, T - 1]
    loud = rand(G, dk, seed=4)
    for n, p in enumerate(edges):
        k[p] = (loud * (2.0 + 0.1 * (n % 7))).to(torch.bfloat16)
    q = (q * 0.2 + loud.repeat_interleave(H // G, 0)[None]).to(torch.bfloat16).double()
    scale = 4.0 / dk
    want = R.attention_heads(q, k, v, scale, R.chunk_mask(T, size))
    other = R.attention_heads(q, k, v, scale, R.chunk_mask(T, size + 1))
    if chunk:
        assert float((other - want).abs().max()) > 0.5                # an edge that is off by one would show
    pages = list(range(1, 22))
    pages = [pages[(i * 8) % 21] for i in range(21)]
    kc, vc = paged(k, pages, 23, dev, dt), paged(v, pages, 23, dev, dt)
    bt = torch.tensor([pages + [0] * 3], dtype=torch.int32, device=dev)
    limit = 2e-5 if dt == torch.float32 else 2e-2
    for q0, q1 in ((0, T), (0, 130), (33, 35), (95, 200), (199, 330), (328, 330), (0, 2)):
        lens = torch.tensor([q1], dtype=torch.int32, device=dev)
        cu = torch.tensor([0, q1 - q0], dtype=torch.int32, device=dev)
        got = ops.attention_prefill(q[q0:q1].contiguous().to(dev, dt), kc, vc, bt, lens, cu, q1 - q0, scale, chunk=chunk)
        assert float((got.double().cpu() - want[q0:q1]).abs().max()) <= limit * float(want.abs().max()), (q0, q1)
    at = sorted({p for e in edges for p in (e, e + 1) if p < T} | {0, 1, 200})
    for splits in (1, 3, 8):
        lens = torch.tensor([p + 1 for p in at], dtype=torch.int32, device=dev)
        got = ops.attention_decode(q[at].contiguous().to(dev, dt), kc, vc, bt.expand(len(at), -1).contiguous(), lens, 1, scale, splits=splits,
                                   chunk=chunk)
        assert float((got.double().cpu() - want[at]).abs().max()) <= limit * float(want.abs().max()), splits


@both
@pytest.mark.parametrize("nq,nkv,dk,dv,rot,chunk", [(6, 2, 40, 24, 8, 20), (2, 2, 128, 64, 128, 0), (8, 1, 64, 128, 32, 64), (4, 2, 128, 128, 0, 33)])
@pytest.mark.parametrize("new,append", [(1, True), (3, True), (1, False)])
def test_decode_step_from_the_projection(dev, dt, nq, nkv, dk, dv, rot, chunk, new, append):
    """Preparation, append and attention in one operator: sequences at page and chunk edges, an idle row."""
    lens = [1 + new, 16, 17, 33, 64, 65, 66, 130, 40]
    B, P, eps = len(lens), 9, 1e-4
    lens_t = torch.tensor(lens)
    bt = (torch.arange(B * P).view(B, P) * 5 % (B * P)) + 1
    pos = torch.cat([torch.arange(n - new, n) for n in lens])
    slots = torch.cat([bt[b][torch.arange(n - new, n) // 16] * 16 + torch.arange(n - new, n) % 16 for b, n in enumerate(lens)])
    slots[-new:] = -1                                                  # idle: its result is not looked at, its pages stay
    x = rand(B * new, nq * dk + (nkv * (dk + dv) if append else 0), seed=1)
    qw, kw = rand(nq * dk, seed=2) * 0.3 + 1, rand(nkv * dk, seed=3) * 0.3 + 1
    inv = torch.tensor([100.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float32)
    k0, v0 = rand(B * P + 1, nkv, 16, dk, seed=4), rand(B * P + 1, nkv, 16, dv, seed=5)
    kr, vr = k0.float(), v0.float()
    q = ops.qkv_prepare_ref(x.float(), pos, slots, inv, kr, vr, nq, nkv, dk, dv, qw.float(), kw.float(), eps, True, append)
    want = ops.attention_ref(q, kr, vr, bt, lens_t, [new] * B, 0.2, chunk=chunk)
    for splits in (1, 4, 8):
        kc, vc = k0.to(dev, dt), v0.to(dev, dt)
        got = ops.attention_decode_rope(x.to(dev, dt), kc, vc, bt.int().to(dev), lens_t.int().to(dev), new, 0.2, pos.int().to(dev), slots.to(dev),
                                        inv.to(dev), nq, nkv, dk, q_norm_w=qw.float().to(dev), k_norm_w=kw.float().to(dev), norm_eps=eps, splits=splits,
                                        chunk=chunk, value_dim=dv, norm_whole=True, value_norm=True, append=append)
        close(got[:-new], want[:-new], dt, scale=float(want.abs().max()) * (3 if dt == torch.bfloat16 else 1))
        close(kc, kr, dt)
        close(vc, vr, dt)


def ragged(rows, starts, pages, dev):
    """ForwardBatch of portions: sequence i brings rows[i] tokens from position starts[i]; its first page is pages[i]."""
    cu = torch.tensor([0] + rows).cumsum(0)
    slots = torch.cat([torch.arange(r) + pages[i] * 16 for i, r in enumerate(rows)])
    return ForwardBatch(token_ids=torch.zeros(int(cu[-1]), dtype=torch.int32, device=dev), positions=torch.zeros(int(cu[-1]), dtype=torch.int32),
                        slots=slots.to(dev), block_table=torch.tensor([[p, 0] for p in pages], dtype=torch.int32, device=dev),
                        seq_lens=torch.tensor([s + r for s, r in zip(starts, rows)], dtype=torch.int32, device=dev),
                        is_prefill=True, cu_q=cu.int().to(dev), max_q_len=max(rows))


PORTIONS = [[300], [1] * 12 + [40, 2, 2, 100, 64, 65, 15], [64, 128, 16, 8, 9, 75]]


def run_portions(step, T, portions):
    outs, at, i = [], 0, 0
    while at < T:
        n = min(portions[min(i, len(portions) - 1)], T - at)
        outs.append(step(at, at + n))
        at, i = at + n, i + 1
    return torch.cat(outs)


@both
@pytest.mark.parametrize("portions", PORTIONS)
@pytest.mark.parametrize("width", [33, 72, 256])
def test_mingru_recurrence(dev, dt, width, portions):
    T = 300
    x = rand(T, 3 * width, seed=1) * 2
    x[:, :width] -= 2                                                 # slow gates: what was seen long ago still counts
    x[0, width:2 * width] += 30
    x = x.to(torch.bfloat16).double()
    z, u = torch.sigmoid(x[:, :width]), x[:, width:2 * width]
    cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    S, want = torch.zeros(width, dtype=torch.float64), []
    for t in range(T):
        S = (1 - z[t]) * S + z[t] * cand[t]
        want.append(S * x[t, 2 * width:] * torch.sigmoid(x[t, 2 * width:]))
    state = torch.zeros(3, width, device=dev)
    p2s = torch.tensor([0, 0, 2, 1], dtype=torch.int32, device=dev)
    got = run_portions(lambda a, b: ops.mingru_scan(x[a:b].contiguous().to(dev, dt), state, width, ragged([b - a], [a], [2], dev), p2s), T, portions)
    close(got, torch.stack(want), dt)
    close(state[2], S, torch.float32, scale=float(S.abs().max()) * 5)
    assert not state[0].any() and not state[1].any()


def gla_inputs(T, H, D, V, rank, seed, strong=False):
    x = rand(T, 2 * H * D + 2 * H * V + rank, seed=seed)
    a2, b = rand(H * D, rank, seed=seed + 1) * 0.3, rand(H * D, seed=seed + 2) * 2 + 2
    if strong:                                                        # some channels forget within a few tokens, others never
        b[::3] -= 30
        b[1::3] += 20
    return x, a2, b, rand(V, seed=seed + 3) * 0.3 + 1


def gla_reference(x, a2, b, nw, H, D, V, tau, eps, S):
    T, qk, vw = x.shape[0], H * D, H * V
    z = (x[:, 2 * qk + 2 * vw:] @ a2.t() + b).view(T, H, D)
    o, S = R.gla_scan(x[:, :qk].view(T, H, D) * D ** -0.5, x[:, qk:2 * qk].view(T, H, D), x[:, 2 * qk:2 * qk + vw].view(T, H, V),
                      torch.sigmoid(z) ** (1.0 / tau), S)
    g = x[:, 2 * qk + vw:2 * qk + 2 * vw]
    return (R.rms(o, eps) * nw).reshape(T, vw) * g * torch.sigmoid(g), S


@both
@pytest.mark.parametrize("portions", PORTIONS)
@pytest.mark.parametrize("H,D,V,rank,tau,strong", [(3, 24, 40, 8, 4.0, False), (2, 64, 128, 16, 16.0, False), (1, 128, 256, 8, 1.0, True),
                                                   (2, 16, 64, 24, 1.0, True), (1, 20, 300, 8, 2.0, False), (1, 12, 10, 3, 2.0, True)])
def test_gated_linear_attention(dev, dt, H, D, V, rank, tau, strong, portions):
    T = 300
    x, a2, b, nw = gla_inputs(T, H, D, V, rank, 7, strong)
    want, S = gla_reference(x, a2, b, nw, H, D, V, tau, 1e-5, torch.zeros(H, D, V, dtype=torch.float64))
    state = torch.zeros(2, H, D, V, device=dev)
    p2s = torch.tensor([0, 1, 0], dtype=torch.int32, device=dev)
    f = lambda t: t.float().to(dev)                                                    # noqa: E731
    got = run_portions(lambda i, j: ops.gla_attention(x[i:j].contiguous().to(dev, dt), f(a2), f(b), f(nw), state, H, D, V, tau, 1e-5,
                                                      ragged([j - i], [i], [1], dev), p2s), T, portions)
    close(got, want, dt)
    close(state[1], S, torch.float32, scale=float(S.abs().max()) * (5 if dt == torch.float32 else 10))      # the state is fp32 in both
    assert not state[0].any()


@both
def test_recurrences_of_a_ragged_batch_and_idle_rows(dev, dt):
    """Portions of unequal length side by side give what each gives alone; a row without a cache slot keeps its state."""
    H, D, V, rank, W = 2, 32, 48, 8, 40
    rows, pages = [70, 1, 130, 2, 64], [3, 1, 5, 2, 4]
    x, a2, b, nw = gla_inputs(sum(rows), H, D, V, rank, 3)
    y = rand(sum(rows), 3 * W, seed=9)
    p2s = torch.tensor([0, 4, 1, 0, 3, 2], dtype=torch.int32, device=dev)
    f = lambda t: t.float().to(dev)                                                    # noqa: E731
    gs, ms = f(rand(5, H, D, V, seed=5)), f(rand(5, W, seed=6))
    gs0, ms0 = gs.clone(), ms.clone()
    batch = ragged(rows, [9] * 5, pages, dev)
    gla = lambda t, s, bt: ops.gla_attention(t.to(dev, dt), f(a2), f(b), f(nw), s, H, D, V, 4.0, 1e-5, bt, p2s)     # noqa: E731
    got_g, got_m = gla(x, gs, batch), ops.mingru_scan(y.to(dev, dt), ms, W, batch, p2s)
    at = 0
    for i, n in enumerate(rows):
        g1, m1 = gs0.clone(), ms0.clone()
        alone = ragged([n], [9], [pages[i]], dev)
        close(got_g[at:at + n], gla(x[at:at + n].contiguous(), g1, alone).double().cpu(), dt)
        close(got_m[at:at + n], ops.mingru_scan(y[at:at + n].contiguous().to(dev, dt), m1, W, alone, p2s).double().cpu(), dt)
        slot = int(p2s[pages[i]])
        close(gs[slot], g1[slot].double().cpu(), torch.float32)
        close(ms[slot], m1[slot].double().cpu(), torch.float32)
        at += n
    B = 5
    idle = ForwardBatch(token_ids=None, positions=None, slots=torch.tensor([5, -1, 9, -1, 3], device=dev), block_table=batch.block_table,
                        seq_lens=batch.seq_lens, is_prefill=False, q_per_seq=1)
    gs, ms = gs0.clone(), ms0.clone()
    gla(x[:B].contiguous(), gs, idle)
    ops.mingru_scan(y[:B].contiguous().to(dev, dt), ms, W, idle, p2s)
    for i in range(B):
        slot = int(p2s[pages[i]])
        assert torch.equal(gs[slot], gs0[slot]) == (i in (1, 3)) and torch.equal(ms[slot], ms0[slot]) == (i in (1, 3))


# ---------------------------------------------------------------------------------------------- whole models
@both
@pytest.mark.parametrize("cfg", [MIXED, ODD], ids=["mixed", "odd"])
def test_prompt_portions_and_decoding_agree_with_the_restatement(dev, dt, cfg):
    w = R.weights(cfg, seed=1)
    tokens = prompt(150, cfg["vocab"], 2)
    want = R.forward(cfg, w, tokens)
    eng = engine_for(cfg, w, dev, dt, max_seq_len=160, num_pages=11, state_slots=1)      # room for one: every run reuses it
    for sizes in ([150], [100, 1], [2, 3, 2, 17, 64], [37, 20, 43, 50], [1]):
        seq = eng.open_sequence()
        got = feed(eng, seq, tokens, sizes)
        assert R.error(got, want) < LIMIT[dt], sizes
        eng.release(seq)


@both
def test_first_tokens_and_one_token_prompts(dev, dt):
    w = R.weights(MIXED, seed=3)
    eng = engine_for(MIXED, w, dev, dt)
    for n in (1, 2, 3, 16, 17):
        tokens = prompt(n, MIXED["vocab"], n)
        seq = eng.open_sequence()
        assert R.error(feed(eng, seq, tokens, [n]), R.forward(MIXED, w, tokens)) < LIMIT[dt]
        eng.release(seq)


@both
def test_a_wrong_mask_or_a_lost_state_would_show(dev, dt):
    """The same comparison with a mistake planted in the restatement is far outside the limit."""
    w = R.weights(MIXED, seed=1)
    tokens = prompt(90, MIXED["vocab"], 2)
    eng = engine_for(MIXED, w, dev, dt)
    got = feed(eng, eng.open_sequence(), tokens, [90])
    for layer, change in ((1, {"mask": {"size": 38}}), (2, {"mask": {"size": 37}}), (2, {"scale": 0.8}), (4, {"rot": {"dims": 126, "base": 50.0}, "scale": 0.2}),
                          (0, {"tau": 8.0})):
        other = json.loads(json.dumps(MIXED))
        other["layers"][layer]["mixer"].update(change)
        assert R.error(got, R.forward(other, w, tokens)) > 2 * LIMIT[dt], (layer, change)


@both
def test_mixed_batches_and_reused_pages(dev, dt):
    """Requests of unequal length in portions beside single decoded tokens; pages and slots run out and are used again."""
    w = R.weights(MIXED, seed=4)
    lengths = [120, 5, 64, 33, 90, 17, 1, 48]
    reqs = [prompt(n, MIXED["vocab"], 10 + i) for i, n in enumerate(lengths)]
    want = [R.forward(MIXED, w, r) for r in reqs]
    eng = engine_for(MIXED, w, dev, dt, max_batch=3, max_seq_len=128, num_pages=20, state_slots=3)
    g = torch.Generator().manual_seed(5)
    live, waiting, got = {}, list(range(len(reqs))), {i: [] for i in range(len(reqs))}
    while live or waiting:
        while waiting and len(live) < 3:
            live[waiting.pop(0)] = [eng.open_sequence(), 0]
        entries, step = [], []
        for i in list(live):
            if len(live) > 1 and int(torch.randint(0, 4, (1,), generator=g)) == 0:
                continue                                              # left out of this step
            seq, at = live[i]
            n = min([1, 1, 2, 7, 40][int(torch.randint(0, 5, (1,), generator=g))], len(reqs[i]) - at)
            entries.append((seq, reqs[i][at:at + n], range(n)))
            step.append((i, n))
        if not entries:
            continue
        logits = eng.forward_tokens(entries)
        at = 0
        for i, n in step:
            got[i].append(logits[at:at + n])
            at += n
            live[i][1] += n
            if live[i][1] == len(reqs[i]):
                eng.release(live.pop(i)[0])
    for i in range(len(reqs)):
        assert R.error(torch.cat(got[i]), want[i]) < LIMIT[dt], i
    assert eng.kv.allocator.free_pages() == 19 and len(eng.kv._free_state_slots) == 3


@both
def test_long_decoding_across_chunks(dev, dt):
    w = R.weights(SMALL, seed=6)
    tokens = prompt(330, SMALL["vocab"], 7)
    eng = engine_for(SMALL, w, dev, dt, max_seq_len=336)
    got = feed(eng, eng.open_sequence(), tokens, [30, 1])
    assert R.error(got, R.forward(SMALL, w, tokens)) < LIMIT[dt]


# ---------------------------------------------------------------------------------------------- generation
def agrees_greedily(cfg, w, prompts, outs, dt):
    """Every generated token is the restatement's choice given what came before it, or so close to it that rounding decides."""
    for p, o in zip(prompts, outs):
        logits = R.forward(cfg, w, p + o)[len(p) - 1:-1]
        chosen = logits.gather(1, torch.tensor(o)[:, None])[:, 0]
        slack = (1e-3 if dt == torch.float32 else 0.3) * float(logits.std())
        assert float((logits.max(-1).values - chosen).max()) <= slack


@both
def test_greedy_generation_through_engine_and_server(dev, dt):
    from eredu_b200.runtime.server import Server

    w = R.weights(MIXED, seed=8)
    prompts = [prompt(n, MIXED["vocab"], n) for n in (3, 41, 18, 70, 9)]
    eng = engine_for(MIXED, w, dev, dt, max_batch=5, max_seq_len=128, prefill_chunk=50)
    sp = SamplingParams(temperature=0.0)
    outs = eng.generate(prompts, sp, max_new_tokens=24)
    agrees_greedily(MIXED, w, prompts, outs, dt)
    assert [len(o) for o in outs] == [24] * 5
    srv = Server(engine_for(MIXED, w, dev, dt, max_batch=3, max_seq_len=128), prefill_chunk=16, max_step_tokens=40)
    ids = [srv.submit(p, sp, 12 + i) for i, p in enumerate(prompts[:3])]
    for _ in range(4):
        srv.step()
    ids += [srv.submit(p, sp, 15 + i) for i, p in enumerate(prompts[3:])]
    srv.run_until_idle(max_steps=400)
    served = [srv.result(i).tokens for i in ids]
    agrees_greedily(MIXED, w, prompts, served, dt)
    if dt == torch.float32:
        assert all(s == o[:len(s)] for s, o in zip(served, outs))


@both
def test_a_request_held_back_for_a_step_keeps_its_state(dev, dt):
    w = R.weights(SMALL, seed=9)
    prompts = [prompt(n, SMALL["vocab"], n) for n in (20, 11)]
    eng = engine_for(SMALL, w, dev, dt, max_batch=2, max_seq_len=96)
    sp = SamplingParams(temperature=0.0)
    want = [eng.generate([p], sp, max_new_tokens=10)[0] for p in prompts]
    seqs = [eng.new_sequence(p, sp, 10) for p in prompts]
    first = eng.prefill(seqs).tolist()
    eng.open_decode()
    for s, t in zip(seqs, first):
        s.output.append(t)
        eng.join(s, t)
    for step in range(40):
        mask = [not s.finished and (step % 3 != 1 or i == 0) and (step % 4 != 2 or i == 1) for i, s in enumerate(seqs)]
        if all(s.finished for s in seqs):
            break
        eng.set_step_mask(mask)
        eng._decode_state["stepped"] = mask
        eng.commit(eng.decode_step().tolist())
    if dt == torch.float32:
        assert [s.output for s in seqs] == want
    agrees_greedily(SMALL, w, prompts, [s.output for s in seqs], dt)


def save(tmp_path, cfg, w):
    from eredu_b200.formats import checkpoint as ck

    mc = ModelConfig.from_hf_dict(cfg)
    ck.save_safetensors_checkpoint(tmp_path, mc, w, torch.bfloat16)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    return mc


@both
def test_checkpoint_loading_inspection_and_trace(dev, dt, tmp_path):
    from eredu_b200.api import LoadedModel, ModelLoadOptions
    from eredu_b200.runtime import trace_replay
    from eredu_b200.runtime.plan import estimate_runtime_state, inspect_artifact

    w = R.weights(MIXED, seed=10, rank=5)                             # a rank that is not a multiple of 8
    mc = save(tmp_path / "m", MIXED, w)
    report = inspect_artifact(tmp_path / "m")
    assert report.is_loadable and report.model_type == "nidozen"
    prof = estimate_runtime_state(mc)
    assert prof.kv_bytes_per_token == 2 * (2 * 64 + 2 * 256 + 88) and prof.state_bytes_per_sequence == 4 * (3 * 24 * 40 + 72)
    lm = LoadedModel.load(tmp_path / "m", ModelLoadOptions(device=dev, dtype=dt, max_batch=2, max_seq_len=96))
    p = prompt(30, MIXED["vocab"], 1)
    assert R.error(lm.prefill_logits(p)[None], R.forward(MIXED, w, p)[-1:]) < LIMIT[dt]
    agrees_greedily(MIXED, w, [p], lm.generate([p], SamplingParams(temperature=0.0), 8), dt)
    eng = trace_replay.load(str(tmp_path / "m"), str(dt).split(".")[1], 128, 2, device=dev).engine
    toks = {"a": prompt(40, MIXED["vocab"], 2), "b": prompt(21, MIXED["vocab"], 3)}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks["a"][:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks["a"][30:31], "want": [0]}, {"id": "b", "tokens": toks["b"][:20], "want": [19]}]},
             {"step": 2, "entries": [{"id": "a", "tokens": toks["a"][31:], "want": []}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": toks["b"][20:], "want": [0]}], "end": ["b"]}]
    done = []
    trace_replay.replay(eng, [json.dumps(s) for s in steps], tmp_path, done.append)
    assert done == [0, 1, 2, 3] and not (tmp_path / "2.f32").exists()
    fa, fb = R.forward(MIXED, w, toks["a"]), R.forward(MIXED, w, toks["b"])
    for step, rows in ((0, fa[[0, 29]]), (1, torch.stack((fa[30], fb[19]))), (3, fb[20:21])):
        got = torch.frombuffer(bytearray((tmp_path / f"{step}.f32").read_bytes()), dtype=torch.float32).view(-1, MIXED["vocab"])
        assert R.error(got, rows) < LIMIT[dt]
    assert eng.kv.allocator.free_pages() == 8


def test_prompt_cache_keeps_pages_and_states(tmp_path):
    from eredu_b200.runtime.prompt_cache import load_prompt_cache, save_prompt_cache

    w = R.weights(MIXED, seed=11)
    p = prompt(45, MIXED["vocab"], 4)
    eng = engine_for(MIXED, w, "cpu", torch.float32)
    seq = eng.new_sequence(p[:40], max_new_tokens=1)
    eng.prefill([seq])
    save_prompt_cache(eng, seq, tmp_path / "c", "fp")
    other = engine_for(MIXED, w, "cpu", torch.float32)
    back = load_prompt_cache(other, tmp_path / "c", p, "fp", max_new_tokens=2)
    assert back.kv_len == 40
    got = other.forward_tokens([(back, p[40:], range(5))])
    assert R.error(got, R.forward(MIXED, w, p)[40:]) < LIMIT[torch.float32]


def test_command_line_generates(tmp_path, capsys):
    from eredu_b200.cli.main import main
    from test_text_streaming import make_bundle

    cfg = dict(SMALL, vocab=make_bundle(tmp_path).vocab_size())
    save(tmp_path, cfg, R.weights(cfg, seed=12))
    tel = tmp_path / "tel.json"
    assert main(["-m", str(tmp_path), "hello", "--device", "cpu", "-n", "6", "--timing", "--telemetry-json", str(tel)]) == 0
    t = json.loads(tel.read_text())
    assert 0 < t["generated_tokens"] <= 6 and t["plan"]["model_type"] == "nidozen" and "TTFT" in capsys.readouterr().err
