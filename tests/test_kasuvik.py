"""Kasuvik: every mechanism alone and whole models against the plain restatement in kasuvik_reference.py - prompts, decoding, portions,
unequal batches, reused pages and slots, window and block edges, greedy generation through the engine and the server."""
import json
import math

import pytest
import torch

import kasuvik_reference as R
from eredu_b200 import ops
from eredu_b200.models.config import ModelConfig
from eredu_b200.models.llama import ForwardBatch, build_from_tensors
from eredu_b200.ops import SamplingParams
from eredu_b200.runtime.engine import Engine

CASES = [pytest.param("cpu", torch.float32, id="cpu-fp32"), pytest.param("cuda", torch.float32, marks=pytest.mark.gpu, id="gpu-fp32"),
         pytest.param("cuda", torch.bfloat16, marks=pytest.mark.gpu, id="gpu-bf16")]
both = pytest.mark.parametrize("dev,dt", CASES)

# Sizes that are unequal where they can be; windows and blocks that end inside pages and on them; layers with and without a feed-forward.
MIXED = R.config(96, 211, [R.parallel_layer(6, 2, 24, 40, 37, 5, 72, 20, 10, 88, conv=2, mamba_conv=3, rot=16, base=1000.0, scale=0.3),
                           R.delta_layer(3, 40, 56),
                           R.parallel_layer(2, 2, 72, 128, 16, 16, 104, 8, 24, 0, conv=4, mamba_conv=2, rot=72, base=500.0, scale=0.1),
                           R.delta_layer(2, 64),
                           R.parallel_layer(4, 1, 128, 16, 50, 33, 64, 130, 8, 40, conv=3, mamba_conv=4, rot=8, base=20000.0, scale=0.15)], eps=3e-5, scale=7.0)
# Sizes the tensor-core kernels do not take (not multiples of 8, odd widths), single heads and states, one tap, blocks and windows of one.
ODD = R.config(70, 97, [R.parallel_layer(3, 1, 9, 13, 7, 1, 33, 5, 3, 51, conv=1, mamba_conv=5, rot=4, base=100.0, scale=0.4),
                        R.delta_layer(3, 7, 13),
                        R.parallel_layer(1, 1, 12, 5, 1, 3, 10, 1, 1, 0, conv=5, mamba_conv=1, rot=2),
                        R.delta_layer(1, 20),
                        R.parallel_layer(4, 2, 16, 8, 20, 2, 24, 16, 7, 30, conv=2, mamba_conv=2, rot=0, scale=0.25)])
SMALL = R.config(64, 97, [R.delta_layer(2, 24, 48), R.parallel_layer(4, 2, 32, 24, 40, 7, 48, 12, 8, 72), R.delta_layer(1, 56)], scale=8.0)
LIMIT = {torch.float32: 3e-4, torch.bfloat16: 0.07}


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


def rand(*shape, seed=0):
    """Random values exact in bf16, on the CPU in fp64."""
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)).to(torch.bfloat16).double()


def close(got, want, dt, scale=None, limit=None):
    got, want = got.double().cpu(), want.double()
    assert got.shape == want.shape
    if not want.numel():
        return
    s = scale or float(want.abs().max())
    limit = limit or (2e-5 if dt == torch.float32 else 1.2e-2)
    assert float((got - want).abs().max()) <= limit * s, float((got - want).abs().max()) / s


def batch_of(portions, tables, dev, prefill=True, most=0):
    """ForwardBatch over the given page lists: portions [(first new position, new tokens)]; ``prefill`` False: a decode step."""
    cu = torch.tensor([0] + [n for _, n in portions]).cumsum(0)
    width = max(len(t) for t in tables)
    pos = [torch.arange(a, a + n) for a, n in portions]
    slots = torch.cat([torch.tensor(t)[p // 16] * 16 + p % 16 for t, p in zip(tables, pos)])
    common = dict(token_ids=None, positions=torch.cat(pos).int().to(dev), slots=slots.to(dev),
                  block_table=torch.tensor([t + [0] * (width - len(t)) for t in tables], dtype=torch.int32, device=dev),
                  seq_lens=torch.tensor([a + n for a, n in portions], dtype=torch.int32, device=dev))
    if not prefill:
        return ForwardBatch(**common, is_prefill=False, q_per_seq=portions[0][1], max_kv_len=most)
    return ForwardBatch(**common, is_prefill=True, cu_q=cu.int().to(dev), max_q_len=max(n for _, n in portions), portions=list(portions))


# ---------------------------------------------------------------------------------------------- configuration
def test_config_keeps_every_layer_and_round_trips():
    cfg = ModelConfig.from_hf_dict(MIXED)
    assert cfg.model_type == "kasuvik" and cfg.num_hidden_layers == 5 and cfg.is_hybrid and cfg.vocab_size == 211 and cfg.embedding_scale == 7.0
    assert [cfg.layer_has_kv(i) for i in range(5)] == [True, False, True, False, True]
    assert cfg.layer_kv_dims(0) == (2, 24, 40) and cfg.layer_kv_dims(4) == (1, 128, 16) and [cfg.layer_kv_pool(i) for i in range(5)] == [5, 0, 16, 0, 33]
    assert cfg.layer_state_shape(1) == (3, 40, 40)
    assert cfg.layer_state_shape(0) == (72 * 20 + 2 * 72 + 1 * (6 * 24 + 2 * 24 + 2 * 40),)
    assert cfg.mixers[0].left.window == 37 and cfg.mixers[0].right.dt_rank == 10 and cfg.mixers[2].ff == 0 and cfg.mixers[4].left.rot_dims == 8
    assert ModelConfig.from_hf_dict(cfg.to_hf_dict()).mixers == cfg.mixers
    for change in ({"type": "attention"}, {"mlp": {"kind": "moe"}}):
        wrong = json.loads(json.dumps(MIXED))
        wrong["layers"][0].update(change)
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(wrong)
    for side, change in (("left", {"kv_heads": 4}), ("left", {"mask": {"size": 0, "pool": 4}}), ("left", {"rot": {"dims": 26, "base": 1.0}}), ("right", {"state": 0})):
        wrong = json.loads(json.dumps(MIXED))
        wrong["layers"][0]["mixer"][side].update(change)
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(wrong)


def test_pooled_rows_lie_beside_the_page_of_their_last_token():
    eng = engine_for(MIXED, R.weights(MIXED), "cpu", torch.float32, state_slots=3)
    assert eng.kv.pooled[0][0].shape[1:] == (2, 4, 24) and eng.kv.pooled[2][1].shape[1:] == (2, 1, 128) and eng.kv.pooled[4][0].shape[1:] == (1, 1, 128)
    assert eng.kv.layer_state[1].shape == (3, 3, 40, 40) and 1 not in eng.kv.pooled
    with pytest.raises(NotImplementedError):
        eng.kv.require_uniform("moving pages")
    for pool in (1, 2, 3, 5, 7, 16, 17, 20, 33, 100):
        seen = set()
        for b in range(400):
            page, row = ops.pooled_row(b, pool)
            assert page * 16 <= b * pool + pool - 1 < page * 16 + 16 and 0 <= row < -(-16 // pool)
            seen.add((page, row))
        assert len(seen) == 400


# ---------------------------------------------------------------------------------------------- mechanisms
@both
@pytest.mark.parametrize("width", [33, 96, 1000, 2500, 8192, 9000])
def test_norms_around_a_sublayer(dev, dt, width):
    M, eps = 5, 1e-4
    x, y0, y1 = (rand(M, width, seed=i) * (i + 0.5) for i in range(3))
    x = x.float()
    y0, y1 = (t.to(torch.bfloat16).double() for t in (y0, y1))
    w0, w1, w, n = (torch.rand(width, generator=torch.Generator().manual_seed(i)) + 0.5 for i in range(4))
    on = lambda t: t.to(dev, dt)                                                        # noqa: E731
    for branches, ws, gain in (([y0], None, 1.0), ([y0, y1], None, 0.7), ([y0, y1], (w0, w1), 0.5), ([y1], (w1,), 2.0)):
        s = gain * sum(y if ws is None else R.rms_norm(y, g, eps) for y, g in zip(branches, ws or branches))
        want = x.double() + R.rms_norm(s, w, eps)
        for nxt in (n, None):
            out, act = ops.branch_norm(x.to(dev), [on(y) for y in branches], w.to(dev), None if nxt is None else nxt.to(dev), eps, dt,
                                       None if ws is None else [g.to(dev) for g in ws], gain)
            close(out, want, torch.float32)
            assert (act is None) == (nxt is None)
            if nxt is not None:
                close(act, R.rms_norm(want, n, eps), dt)


@both
@pytest.mark.parametrize("M,K,N", [(1, 64, 40), (3, 70, 51), (40, 96, 128), (130, 64, 72), (300, 128, 64), (700, 64, 200)])
def test_relu_gated_projection(dev, dt, M, K, N):
    x, w = rand(M, K, seed=1), (rand(2 * N, K, seed=2) / 8).to(torch.bfloat16).double()
    g, u = x @ w[:N].t(), x @ w[N:].t()
    for act, want in (("relu", torch.relu(g) * u), ("silu", R.silu(g) * u)):
        close(ops.gated_linear(x.to(dev, dt), w.to(dev, dt), N, activation=act), want, dt)


CONV = [(6, 2, 24, 40, 16, 72, 2, 3, 5), (2, 2, 72, 128, 72, 104, 4, 2, 16), (4, 1, 128, 16, 8, 64, 3, 4, 33), (3, 1, 9, 13, 4, 33, 1, 5, 1), (1, 1, 12, 5, 2, 10, 5, 1, 3),
        (4, 2, 16, 8, 0, 24, 3, 3, 2), (2, 1, 8, 8, 8, 1100, 4, 6, 20)]


@both
@pytest.mark.parametrize("H,G,dk,dv,rot,width,taps,ctaps,pool", CONV)
def test_convolved_projections(dev, dt, H, G, dk, dv, rot, width, taps, ctaps, pool):
    """Convolution, rotation, temperature and append, and the convolved channels, in one portion, in portions of every kind and token
    by token; the means of the blocks follow."""
    T, base = 150, 300.0
    n, gap = H * dk + G * (dk + dv), 3
    start = n + gap + (-(n + gap) % 8 if dk % 8 == 0 else 0)
    cols = start + width
    cols += -cols % 8
    x = rand(T, cols, seed=1)
    ht, ct = rand(taps, n, seed=2) / taps ** 0.5, rand(ctaps, width, seed=3) / ctaps ** 0.5
    bias, temp = rand(width, seed=4), rand(H, seed=5) + 1.5
    inv = torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float32)
    y = R.causal_conv(x[:, :n], ht.t())
    pos = torch.arange(T)
    q = R.rotate(y[:, :H * dk].view(T, H, dk), pos, base, rot) * temp[None, :, None]
    k = R.rotate(y[:, H * dk:(H + G) * dk].view(T, G, dk), pos, base, rot)
    v = y[:, (H + G) * dk:].view(T, G, dv)
    c = R.silu(R.causal_conv(x[:, start:start + width], ct.t()) + bias)
    table = [(i * 7) % 10 + 1 for i in range(10)]
    hist = (taps - 1) * n
    f = lambda t: t.float().contiguous().to(dev)                                        # noqa: E731
    limit = 1e-4 if dt == torch.float32 else None                                       # angles in fp32
    for sizes in ([T], [1], [40, 1, 1, 2, 3, 64, 5, 34], [2, 1, 7, 90, 17, 33]):
        kc, vc = (torch.zeros(12, G, 16, d, device=dev, dtype=dt) for d in (dk, dv))
        pooled = tuple(torch.zeros(12, G, -(-16 // pool), d, device=dev, dtype=dt) for d in (dk, dv))
        first = 4 if dk % 8 == 0 and taps != 4 else 5                             # histories at whole 16-byte pieces and elsewhere
        state = torch.zeros(3, first + hist + (ctaps - 1) * width + (-(first + hist + (ctaps - 1) * width) % 4 if first == 4 else 0), device=dev)
        state[0] = 9.0
        p2s = torch.zeros(12, dtype=torch.int32, device=dev)
        p2s[table[0]] = 2
        heads = ops.ConvHeads(f(ht), H, G, dk, dv, inv.to(dev), kc, vc, f(temp), pool, pooled, first)
        chans = ops.ConvChannels(f(ct), f(bias), start, first + hist)
        at, i, qs, cs = 0, 0, [], []
        while at < T:
            m = min(sizes[min(i, len(sizes) - 1)], T - at)
            bt = batch_of([(at, m)], [table], dev, prefill=m > 1)
            a, b = ops.conv_project(x[at:at + m].contiguous().to(dev, dt), state, bt, p2s, heads, chans)
            if m > 1 and dev == "cuda":
                ops.pool_blocks(kc, vc, pooled, bt, pool)
            qs.append(a)
            cs.append(b)
            at, i = at + m, i + 1
        close(torch.cat(qs), q, dt, limit=limit)
        close(torch.cat(cs), c, dt)
        t = torch.tensor(table)[pos // 16]
        close(kc[t, :, pos % 16], k, dt, limit=limit)
        close(vc[t, :, pos % 16], v, dt)
        mk, mv = ops.gather_pooled(pooled, bt.block_table[0], T // pool, pool)
        close(mk.transpose(0, 1), R.pooled(k, pool), dt, scale=float(k.abs().max()), limit=limit)
        close(mv.transpose(0, 1), R.pooled(v, pool), dt, scale=float(v.abs().max()))
        st = state[2].double().cpu()
        close(st[first:first + hist].view(taps - 1, n), x[T - taps + 1:, :n], torch.float32, scale=1.0)
        close(st[first + hist:first + hist + (ctaps - 1) * width].view(ctaps - 1, width), x[T - ctaps + 1:, start:start + width], torch.float32, scale=1.0)
        assert bool((state[0] == 9.0).all()) and not state[1].any()
        outside = [p for p in range(12) if p not in table]
        assert not kc[outside].any() and not pooled[0][outside].any()


@both
def test_convolutions_of_a_ragged_batch_and_idle_rows(dev, dt):
    H, G, dk, dv, width, taps, ctaps, pool = 2, 1, 16, 24, 40, 3, 4, 4
    rows, starts = [20, 1, 33, 2, 16, 3], [5, 40, 0, 13, 15, 1]
    tables = [[i * 4 + 1 + j for j in range(4)] for i in range(6)]
    n = H * dk + G * (dk + dv)
    x = rand(sum(rows), n + width, seed=1).to(dev, dt)
    f = lambda t: t.float().contiguous().to(dev)                                        # noqa: E731
    ht, ct, inv = f(rand(taps, n, seed=2)), f(rand(ctaps, width, seed=3)), torch.rand(8, device=dev)
    state0 = f(rand(6, (taps - 1) * n + (ctaps - 1) * width, seed=4))
    p2s = torch.zeros(25, dtype=torch.int32, device=dev)
    for i, slot in enumerate((4, 1, 0, 3, 2, 5)):
        p2s[tables[i][0]] = slot

    def run(x, bt, state):
        kc, vc = (torch.zeros(25, G, 16, d, device=dev, dtype=dt) for d in (dk, dv))
        pooled = tuple(torch.zeros(25, G, 4, d, device=dev, dtype=dt) for d in (dk, dv))
        heads = ops.ConvHeads(ht, H, G, dk, dv, inv, kc, vc, None, pool, pooled, 0)
        return ops.conv_project(x, state, bt, p2s, heads, ops.ConvChannels(ct, None, n, (taps - 1) * n)), kc

    state = state0.clone()
    (q, c), kc = run(x, batch_of(list(zip(starts, rows)), tables, dev), state)
    at = 0
    for i, m in enumerate(rows):
        alone = state0.clone()
        (qa, ca), ka = run(x[at:at + m].contiguous(), batch_of([(starts[i], m)], [tables[i]], dev), alone)
        slot = int(p2s[tables[i][0]])
        assert torch.equal(q[at:at + m], qa) and torch.equal(c[at:at + m], ca) and torch.equal(state[slot], alone[slot])
        assert torch.equal(kc[tables[i]], ka[tables[i]])
        at += m
    bt = batch_of([(s + 1, 1) for s in starts], tables, dev, prefill=False)
    bt.slots = torch.where(torch.tensor([0, 1, 0, 1, 0, 0], device=dev) == 1, -1, bt.slots)
    state = state0.clone()
    _, kc = run(x[:6].contiguous(), bt, state)
    for i in range(6):
        slot = int(p2s[tables[i][0]])
        assert torch.equal(state[slot], state0[slot]) == (i in (1, 3)) and bool(kc[tables[i]].any()) == (i not in (1, 3))


ATTENTION = [(6, 2, 24, 40, 37, 5), (2, 2, 72, 128, 16, 16), (4, 1, 128, 16, 50, 33), (3, 1, 64, 64, 100, 1), (8, 4, 64, 128, 21, 12), (40, 1, 16, 8, 30, 3), (2, 1, 128, 128, 130, 2),
             (3, 1, 9, 13, 7, 2), (1, 1, 136, 40, 1, 20), (4, 4, 32, 24, 2, 7)]


@both
@pytest.mark.parametrize("H,G,dk,dv,window,pool", ATTENTION)
def test_attention_sees_its_window_and_the_blocks_behind_it(dev, dt, H, G, dk, dv, window, pool):
    """Keys at the edges of windows, blocks and pages and the first tokens are made to stand out: one token or block just inside or just
    outside what a query sees decides the row."""
    T, scale = 330, 1.0
    loud = rand(G, dk, seed=9)
    k, v = rand(T, G, dk, seed=1), rand(T, G, dv, seed=2)
    edges = sorted({0, 1, 15, 16, 17, 150, 151, T - 1, T - 2} | set(range(0, T, 37)))
    whole = [p for b in {0, 1, 3, 8, T // pool // 2, T // pool - 2} for p in range(max(0, b) * pool, max(0, b) * pool + pool)]
    for n, p in enumerate(edges + whole):
        if p < T:
            k[p] = k[p] * 0.5 + loud * (1.0 + 0.1 * (n % 5))
    k = k.to(torch.bfloat16).double()
    q = rand(T, H, dk, seed=3) * 0.2 / dk ** 0.5 + (loud * (5.0 / loud.square().sum(-1, keepdim=True))).repeat_interleave(H // G, 0)
    q = q.to(torch.bfloat16).double()
    want = R.pooled_attention(q, k, v, scale, window, pool)
    top = float(want.abs().max())
    others = [(window, pool + 1)] if pool == 1 else [(window, pool + 1), (window + 1, pool)] + ([(window - 1, pool)] if window > 1 else [])
    for other in others:
        assert float((R.pooled_attention(q, k, v, scale, *other) - want).abs().max()) > 0.1 * top       # off by one would show
    table = [(i * 8) % 21 + 1 for i in range(21)]
    pos = torch.arange(T)
    at_page = torch.tensor(table)[pos // 16]
    kc, vc = (torch.full((23, G, 16, d), 3.0, device=dev, dtype=dt) for d in (dk, dv))
    kc[at_page, :, pos % 16], vc[at_page, :, pos % 16] = k.to(dev, dt), v.to(dev, dt)
    row = torch.tensor(table, dtype=torch.int32, device=dev)
    limit = 2e-5 if dt == torch.float32 else 2.5e-2

    def run(portions, prefill=True, most=0):
        pooled = tuple(torch.full((23, G, -(-16 // pool), d), 5.0, device=dev, dtype=dt) for d in (dk, dv))
        start = max(a for a, _ in portions)                          # the sequences share pages: what one of them finds must be there
        for b in range((start if prefill and dev == "cuda" else max(a + n for a, n in portions)) // pool):
            ops.pool_block_ref(kc, vc, pooled, row, b, pool)
        rows = [p for a, n in portions for p in range(a, a + n)]
        y = ops.pooled_attention(q[rows].contiguous().to(dev, dt), kc, vc, pooled, batch_of(portions, [table] * len(portions), dev, prefill, most), scale,
                                 window, pool)
        err = (y.double().cpu() - want[rows]).abs().flatten(1).max(1).values
        assert float(err.max()) <= limit * top, (portions, prefill, rows[int(err.argmax())], float(err.max()) / top)

    for a, b in [(0, T), (0, 130), (33, 35), (95, 200), (199, 330), (328, 330), (0, 2)]:
        run([(a, b - a)])
    run([(0, 140), (0, 1), (0, 200), (0, 31), (0, 9)])
    run([(200, 1), (202, 2), (200, 130), (299, 31)])
    at = sorted({p for e in edges + [b * pool + pool - 1 for b in range(0, T // pool, 5)] for p in (e, e + 1, e + window - 1, e + window, e + window + 1) if p < T})
    for most in (0, T, 4096):                                            # how far a step may see chooses the split of the keys
        run([(p, 1) for p in at], prefill=False, most=most)
    run([(p, 3) for p in at if p + 3 <= T], prefill=False, most=T)
    run([(at[-1], 1)], prefill=False, most=T)


def scan_inputs(T, C, N, rank, seed, kind):
    """"plain"; "keep": tiny steps after a loud start, so the first tokens still count; "swing": steps from none to many time constants."""
    x, z, p = rand(T, C, seed=seed), rand(T, C, seed=seed + 1), rand(T, rank + 2 * N, seed=seed + 2)
    w, b = (rand(C, rank, seed=seed + 3) / rank ** 0.5).to(torch.bfloat16).double(), rand(C, seed=seed + 4) - 2.0
    A, D = -torch.exp(rand(C, N, seed=seed + 5)), rand(C, seed=seed + 6)
    if kind == "keep":
        p[:, :rank] = 0
        b = b - 4.0
        x[:3] *= 20
    elif kind == "swing":
        p[:, :rank] = torch.where(torch.arange(T)[:, None] % 13 == 4, 4.0, -1.0) * p[:, :rank].abs()
        w = w.abs()
        b = b + 1
    exact = lambda t: t.to(torch.bfloat16).double()                                     # noqa: E731
    return exact(x), z, exact(p), w, b, A, D


PORTIONS = [[300], [1] * 12 + [40, 2, 2, 100, 64, 65, 15], [64, 128, 16, 8, 9, 75]]


@both
@pytest.mark.parametrize("portions", PORTIONS)
@pytest.mark.parametrize("C,N,rank,kind", [(72, 20, 8, "plain"), (104, 16, 24, "keep"), (40, 130, 16, "swing"), (33, 5, 3, "swing"), (10, 1, 1, "plain"), (520, 32, 40, "keep"), (128, 16, 40, "swing"),
                                           (48, 32, 8, "plain"), (192, 8, 16, "keep"), (40, 64, 72, "plain")])
def test_selective_scan(dev, dt, C, N, rank, kind, portions):
    T = 300
    x, z, p, w, b, A, D = scan_inputs(T, C, N, rank, 7, kind)
    y, S = R.selective_scan(x, R.softplus(p[:, :rank] @ w.t() + b), p[:, rank:rank + N], p[:, rank + N:], A, D, torch.zeros(C, N, dtype=torch.float64))
    want = y * R.silu(z)
    f = lambda t: t.float().contiguous().to(dev)                                        # noqa: E731
    state = torch.zeros(2, C * N + 4, device=dev)
    p2s = torch.tensor([0, 1, 0], dtype=torch.int32, device=dev)
    pad = -p.shape[1] % 8
    p, zz = torch.cat((p, torch.full((T, pad), 7.0, dtype=torch.float64)), 1), torch.cat((rand(T, 8, seed=1), z), 1)
    outs, at, i = [], 0, 0
    while at < T:
        k = min(portions[min(i, len(portions) - 1)], T - at)
        g = lambda t: t[at:at + k].contiguous().to(dev, dt)                             # noqa: E731
        bt = batch_of([(0, k)], [[1] * 20], dev, prefill=k > 1)
        outs.append(ops.selective_scan(g(x), g(zz)[:, 8:], g(p), rank, w.to(dev, dt).contiguous(), f(b), f(A), f(D), state, bt, p2s))
        at, i = at + k, i + 1
    close(torch.cat(outs), want, dt, limit=1e-4 if dt == torch.float32 else None)
    close(state[1, :C * N].view(C, N), S, torch.float32, limit=1e-4)
    assert not state[0].any() and not state[1, C * N:].any()


@both
def test_selective_scan_of_a_ragged_batch_and_idle_rows(dev, dt):
    C, N, rank = 64, 16, 24
    rows, pages = [200, 1, 130, 2, 64, 17], [3, 1, 5, 2, 4, 6]
    x, z, p, w, b, A, D = scan_inputs(sum(rows), C, N, rank, 3, "plain")
    f = lambda t: t.float().contiguous().to(dev)                                        # noqa: E731
    st0 = f(rand(6, C * N, seed=5))
    p2s = torch.tensor([0, 4, 1, 0, 3, 2, 5], dtype=torch.int32, device=dev)
    g = lambda t, a, e: t[a:e].contiguous().to(dev, dt)                                 # noqa: E731
    step = lambda a, e, st, bt: ops.selective_scan(g(x, a, e), g(z, a, e), g(p, a, e), rank, w.to(dev, dt), f(b), f(A), f(D), st, bt, p2s)     # noqa: E731
    st = st0.clone()
    got, at = step(0, sum(rows), st, batch_of([(0, n) for n in rows], [[q] * 20 for q in pages], dev)), 0
    for i, n in enumerate(rows):
        alone = st0.clone()
        close(got[at:at + n], step(at, at + n, alone, batch_of([(0, n)], [[pages[i]] * 20], dev)).double().cpu(), dt)
        slot = int(p2s[pages[i]])
        close(st[slot], alone[slot].double().cpu(), torch.float32)
        at += n
    idle = batch_of([(0, 1)] * 6, [[q] for q in pages], dev, prefill=False)
    idle.slots = torch.tensor([5, -1, 9, -1, 3, 7], device=dev)
    st = st0.clone()
    step(0, 6, st, idle)
    for i in range(6):
        slot = int(p2s[pages[i]])
        assert torch.equal(st[slot], st0[slot]) == (i in (1, 3))


@both
@pytest.mark.parametrize("C,N,rank", [(64, 16, 24), (96, 8, 8), (24, 64, 16), (40, 12, 5)])
def test_scan_steps_of_many_sequences(dev, dt, C, N, rank):
    """Decode steps of more sequences than a CTA takes, idle rows among them."""
    n = 37
    x, z, p, w, b, A, D = scan_inputs(n, C, N, rank, 3, "plain")
    S0 = rand(n, C, N, seed=5)
    st = torch.zeros(n + 1, C * N + 8, device=dev)
    st[1:, :C * N] = S0.flip(0).reshape(n, -1).float().to(dev)                        # sequence i has slot n - i
    p2s = torch.tensor([0] + [n - i for i in range(n)], dtype=torch.int32, device=dev)
    bt = batch_of([(3, 1)] * n, [[i + 1] for i in range(n)], dev, prefill=False)
    idle = [5, 16, 30]
    bt.slots[idle] = -1
    f = lambda t: t.float().contiguous().to(dev)                                        # noqa: E731
    p = torch.cat((p, torch.zeros(n, -p.shape[1] % 8, dtype=torch.float64)), 1)
    before = st.clone()
    got = ops.selective_scan(x.to(dev, dt), z.to(dev, dt), p.to(dev, dt), rank, w.to(dev, dt).contiguous(), f(b), f(A), f(D), st, bt, p2s)
    for i in range(n):
        if i in idle:
            assert torch.equal(st[n - i], before[n - i])
            continue
        y, S = R.selective_scan(x[i:i + 1], R.softplus(p[i:i + 1, :rank] @ w.t() + b), p[i:i + 1, rank:rank + N], p[i:i + 1, rank + N:rank + 2 * N], A, D, S0[i])
        close(got[i:i + 1], y * R.silu(z[i:i + 1]), dt)
        close(st[n - i, :C * N].view(C, N), S, torch.float32)
    assert not st[0].any() and not st[:, C * N:].any()


def delta_inputs(T, H, dk, dv, rank, seed, kind):
    """"plain"; "keep": little is forgotten and keys repeat, so what is removed and what stays both show; "wipe": strong decay and
    removal; "same": one key again and again."""
    qk = H * dk
    x = rand(T, 3 * qk + 2 * H * dv + rank, seed=seed)
    w2, w0, rb = (rand(qk, rank, seed=seed + 1) / rank ** 0.5).to(torch.bfloat16).double(), rand(qk, seed=seed + 2) - 2, rand(qk, seed=seed + 3)
    keys = x[:, qk:2 * qk]
    if kind == "keep":
        w0 = w0 - 6
        keys.copy_(rand(7, qk, seed=seed + 4)[torch.arange(T) % 7])
    elif kind == "wipe":
        w0, rb = w0 + 8, rb + 4
    elif kind == "same":
        w0 = w0 - 4
        keys.copy_((rand(1, qk, seed=seed + 4) * 0.3).to(torch.bfloat16).expand(T, qk))
        rb = rb + 2
    return x, w2, w0, rb, rand(H * dv, seed=seed + 5) * 0.3 + 1


def delta_reference(x, w2, w0, rb, nw, H, dk, dv, c, eps, state):
    T, qk, vw = x.shape[0], H * dk, H * dv
    r, k, v, g, a, low = torch.split(x, [qk, qk, vw, vw, qk, x.shape[1] - 3 * qk - 2 * vw], 1)
    decay = torch.exp(-c * R.sigmoid(torch.tanh(low) @ w2.t() + w0))
    o, state = R.delta_scan(r.view(T, H, dk), k.view(T, H, dk), v.view(T, H, dv), decay.view(T, H, dk), R.sigmoid(a + rb).view(T, H, dk), state)
    return R.unit_rms(o, eps).reshape(T, vw) * nw * R.sigmoid(g), state


@both
@pytest.mark.parametrize("portions", PORTIONS)
@pytest.mark.parametrize("H,dk,dv,rank,kind,c", [(3, 40, 40, 16, "plain", 0.6), (2, 64, 64, 8, "keep", math.exp(-0.5)), (2, 64, 64, 24, "wipe", math.exp(-0.5)),
                                                 (1, 128, 128, 64, "plain", 0.3), (2, 128, 64, 16, "same", 0.6), (1, 24, 96, 40, "keep", 1.0), (3, 7, 5, 3, "plain", 0.6),
                                                 (1, 132, 140, 8, "keep", 0.6), (2, 16, 16, 8, "same", 0.6), (1, 64, 48, 104, "plain", 0.6), (2, 128, 128, 24, "wipe", 0.6)])
def test_generalised_delta_rule(dev, dt, H, dk, dv, rank, kind, c, portions):
    T = 300
    args = delta_inputs(T, H, dk, dv, rank, 7, kind)
    x = args[0]
    want, S = delta_reference(*args, H, dk, dv, c, 1e-5, torch.zeros(H, dk, dv, dtype=torch.float64))
    f = lambda t: t.float().contiguous().to(dev)                                        # noqa: E731
    state = torch.zeros(2, H, dk, dv, device=dev)
    p2s = torch.tensor([0, 1, 0], dtype=torch.int32, device=dev)
    x = torch.cat((x, torch.full((T, -x.shape[1] % 8), 9.0, dtype=torch.float64)), 1)
    outs, at, i = [], 0, 0
    while at < T:
        k = min(portions[min(i, len(portions) - 1)], T - at)
        outs.append(ops.general_delta(x[at:at + k].contiguous().to(dev, dt), *map(f, args[1:]), state, H, dk, dv, c, 1e-5,
                                      batch_of([(0, k)], [[1] * 20], dev, prefill=k > 1), p2s))
        at, i = at + k, i + 1
    close(torch.cat(outs), want, dt, limit=1e-4 if dt == torch.float32 else None)
    close(state[1], S, torch.float32, limit=1e-4)                       # the state is fp32 in both
    assert not state[0].any()


@both
def test_delta_rule_of_a_ragged_batch_and_idle_rows(dev, dt):
    H, dk, dv, rank, c = 2, 32, 48, 8, 0.6
    rows, pages = [70, 1, 130, 2, 64, 17], [3, 1, 5, 2, 4, 6]
    args = delta_inputs(sum(rows), H, dk, dv, rank, 3, "plain")
    f = lambda t: t.float().contiguous().to(dev)                                        # noqa: E731
    st0 = f(rand(6, H, dk, dv, seed=5))
    p2s = torch.tensor([0, 4, 1, 0, 3, 2, 5], dtype=torch.int32, device=dev)
    step = lambda a, e, st, bt: ops.general_delta(args[0][a:e].contiguous().to(dev, dt), *map(f, args[1:]), st, H, dk, dv, c, 1e-5, bt, p2s)     # noqa: E731
    st = st0.clone()
    got, at = step(0, sum(rows), st, batch_of([(0, n) for n in rows], [[q] * 20 for q in pages], dev)), 0
    for i, n in enumerate(rows):
        alone = st0.clone()
        close(got[at:at + n], step(at, at + n, alone, batch_of([(0, n)], [[pages[i]] * 20], dev)).double().cpu(), dt)
        slot = int(p2s[pages[i]])
        close(st[slot], alone[slot].double().cpu(), torch.float32, limit=1e-4)
        at += n
    idle = batch_of([(0, 1)] * 6, [[q] for q in pages], dev, prefill=False)
    idle.slots = torch.tensor([5, -1, 9, -1, 3, 7], device=dev)
    st = st0.clone()
    step(0, 6, st, idle)
    for i in range(6):
        slot = int(p2s[pages[i]])
        assert torch.equal(st[slot], st0[slot]) == (i in (1, 3))


# ---------------------------------------------------------------------------------------------- whole models
def agrees(got, want, dt, slack=1.0):
    e = R.errors(got, want)
    assert float(e.max()) < slack * LIMIT[dt], (float(e.max()), int(e.argmax()))


@both
@pytest.mark.parametrize("cfg", [MIXED, ODD], ids=["mixed", "odd"])
def test_prompt_portions_and_decoding_agree_with_the_restatement(dev, dt, cfg):
    w = R.weights(cfg, seed=1)
    tokens = prompt(150, cfg["vocab"], 2)
    want = R.forward(cfg, w, tokens)
    eng = engine_for(cfg, w, dev, dt, max_seq_len=160, num_pages=11, state_slots=1)      # room for one: every run reuses it
    for sizes in ([150], [100, 1], [2, 3, 2, 17, 64], [37, 20, 43, 50], [1]):
        seq = eng.open_sequence()
        agrees(feed(eng, seq, tokens, sizes), want, dt, 3.0 if cfg is ODD and dt == torch.bfloat16 else 1.0)   # narrow layers amplify rounding
        eng.release(seq)


@both
def test_residual_stream_of_every_layer(dev, dt):
    from eredu_b200.runtime.inspection import ActivationObserver

    class Watch(ActivationObserver):
        def __init__(self):
            self.outputs, self.zero = {}, None

        def observe(self, name, value):
            self.outputs[name] = value.detach().double().cpu()

        def intervene(self, name, value):
            return value * 0 if name == self.zero else None

    w = R.weights(MIXED, seed=12)
    tokens = prompt(70, MIXED["vocab"], 5)
    want, layers = R.forward(MIXED, w, tokens, return_layers=True)
    eng = engine_for(MIXED, w, dev, dt)
    eng.model.observer = watch = Watch()
    agrees(feed(eng, eng.open_sequence(), tokens, [70]), want, dt)
    for i, x in enumerate(layers):
        close(watch.outputs[f"model.layers.{i}.output"], x, dt, limit=1e-4 if dt == torch.float32 else 3e-2)
    watch.zero = "model.layers.3.output"                                  # a stream somebody replaced is what the next layer reads
    assert R.error(feed(eng, eng.open_sequence(), tokens, [70]), want) > 0.1


@both
def test_first_tokens_and_one_token_prompts(dev, dt):
    w = R.weights(MIXED, seed=3)
    eng = engine_for(MIXED, w, dev, dt)
    for n in (1, 2, 3, 16, 17):
        tokens = prompt(n, MIXED["vocab"], n)
        seq = eng.open_sequence()
        agrees(feed(eng, seq, tokens, [n]), R.forward(MIXED, w, tokens), dt)
        eng.release(seq)


@both
def test_a_planted_mistake_would_show(dev, dt):
    """The same comparison with a mistake planted in the restatement is far outside the limit."""
    w = R.weights(MIXED, seed=1)
    tokens = prompt(90, MIXED["vocab"], 2)
    eng = engine_for(MIXED, w, dev, dt)
    got = feed(eng, eng.open_sequence(), tokens, [90])
    for layer, side, change in ((0, "left", {"mask": {"size": 38, "pool": 5}}), (0, "left", {"mask": {"size": 36, "pool": 5}}), (0, "left", {"mask": {"size": 37, "pool": 11}}),
                                (2, "left", {"mask": {"size": 17, "pool": 16}}), (2, "left", {"scale": 0.2}), (4, "left", {"rot": {"dims": 16, "base": 20000.0}}),
                                (2, "left", {"rot": {"dims": 72, "base": 50.0}})):
        other = json.loads(json.dumps(MIXED))
        other["layers"][layer]["mixer"][side].update(change)
        assert R.error(got, R.forward(other, w, tokens)) > 1.5 * LIMIT[dt], (layer, change)
    for name, factor in (("l0.mix.left.temp", 0.5), ("l0.mix.left.k.b", 0.0), ("l0.mix.right.conv.b", 0.0), ("l0.mix.right.D", 0.0), ("l0.mix.right.dt.b", 0.0),
                         ("l1.mix.a.b", -1.0), ("l1.mix.w0", -1.0), ("l1.mix.w2", 0.0), ("l0.norm1b", 0.5), ("l2.mix.left.out", 0.0)):
        other = dict(w, **{name: w[name] * factor})
        assert R.error(got, R.forward(MIXED, other, tokens)) > 1.5 * LIMIT[dt], name


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
        agrees(torch.cat(got[i]), want[i], dt)
    assert eng.kv.allocator.free_pages() == 19 and len(eng.kv._free_state_slots) == 3


@both
def test_long_decoding_across_windows_and_blocks(dev, dt):
    w = R.weights(SMALL, seed=6)
    tokens = prompt(330, SMALL["vocab"], 7)
    eng = engine_for(SMALL, w, dev, dt, max_seq_len=336)
    agrees(feed(eng, eng.open_sequence(), tokens, [30, 1]), R.forward(SMALL, w, tokens), dt)


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
    outs = eng.generate(prompts, sp, max_new_tokens=40)
    agrees_greedily(MIXED, w, prompts, outs, dt)
    assert [len(o) for o in outs] == [40] * 5
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

    w = R.weights(MIXED, seed=10)
    mc = save(tmp_path / "m", MIXED, w)
    report = inspect_artifact(tmp_path / "m")
    assert report.is_loadable and report.model_type == "kasuvik"
    prof = estimate_runtime_state(mc)
    page = 2 * (2 * 64 * 20 + 2 * 200 * 17 + 144 * 17)
    assert prof.kv_bytes_per_token == -(-page // 16)
    assert prof.state_bytes_per_sequence == 4 * sum(math.prod(mc.layer_state_shape(i)) for i in range(5))
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


def test_prompt_cache_keeps_pages_means_and_states(tmp_path):
    from eredu_b200.runtime.prompt_cache import load_prompt_cache, save_prompt_cache

    w = R.weights(MIXED, seed=11)
    p = prompt(120, MIXED["vocab"], 4)
    eng = engine_for(MIXED, w, "cpu", torch.float32)
    seq = eng.new_sequence(p[:100], max_new_tokens=1)
    eng.prefill([seq])
    save_prompt_cache(eng, seq, tmp_path / "c", "fp")
    other = engine_for(MIXED, w, "cpu", torch.float32)
    back = load_prompt_cache(other, tmp_path / "c", p, "fp", max_new_tokens=2)
    assert back.kv_len == 100
    got = other.forward_tokens([(back, p[100:], range(20))])
    assert R.error(got, R.forward(MIXED, w, p)[100:]) < LIMIT[torch.float32]


def test_command_line_generates(tmp_path, capsys):
    from eredu_b200.cli.main import main
    from test_text_streaming import make_bundle

    cfg = dict(SMALL, vocab=make_bundle(tmp_path).vocab_size())
    save(tmp_path, cfg, R.weights(cfg, seed=12))
    tel = tmp_path / "tel.json"
    assert main(["-m", str(tmp_path), "hello", "--device", "cpu", "-n", "6", "--timing", "--telemetry-json", str(tel)]) == 0
    t = json.loads(tel.read_text())
    assert 0 < t["generated_tokens"] <= 6 and t["plan"]["model_type"] == "kasuvik" and "TTFT" in capsys.readouterr().err


def test_random_models_of_a_configuration():
    from eredu_b200.models.llama import build_random, random_state

    mc = ModelConfig.from_hf_dict(SMALL)
    sd = random_state(mc, seed=3)
    a, b = build_from_tensors(mc, sd.__getitem__, sd.__contains__, "cpu", torch.float32), build_random(mc, "cpu", torch.float32, seed=3)
    assert torch.equal(a.layers[1].extra["x"], b.layers[1].extra["x"]) and a.weight_bytes() > 0
    assert Engine(a, max_batch=1, max_seq_len=64).generate([[1, 2, 3]], SamplingParams(temperature=0.0), 4) == \
        Engine(b, max_batch=1, max_seq_len=64).generate([[1, 2, 3]], SamplingParams(temperature=0.0), 4)
