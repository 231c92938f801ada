"""Lenitar: every mechanism alone and whole models against the plain restatement in lenitar_reference.py - prompts, decoding,
portions, unequal batches, reused pages and slots, window edges, sinks, routing, greedy generation through the engine and the server."""
import json
import math

import pytest
import torch

import lenitar_reference as R
from eredu_b200 import ops
from eredu_b200.models.config import ModelConfig
from eredu_b200.models.llama import ForwardBatch, build_from_tensors
from eredu_b200.ops import SamplingParams
from eredu_b200.ops import latent as latent_ops
from eredu_b200.ops import moe as moe_ops
from eredu_b200.runtime.engine import Engine

CASES = [pytest.param("cpu", torch.float32, id="cpu-fp32"), pytest.param("cuda", torch.float32, marks=pytest.mark.gpu, id="gpu-fp32"),
         pytest.param("cuda", torch.bfloat16, marks=pytest.mark.gpu, id="gpu-bf16")]
both = pytest.mark.parametrize("dev,dt", CASES)

# Sizes that are unequal where they can be; windows that end inside pages and on them; layers with and without experts. Every token
# uses all experts of a layer, so that rounding cannot change a choice and each position can be compared.
MIXED = R.config(96, 211, [R.latent(3, 16, 8, 24, 40, 56, 37, R.moe(3, 3, 40), 1000.0, 0.3), R.mlstm_layer(2, 24, 40, 9.0, R.moe(2, 2, 72, 2, 2)),
                           R.latent(5, 64, 32, 48, 64, 24, 16, None, 20000.0, 0.15), R.mlstm_layer(3, 16, 136, 15.0),
                           R.latent(2, 72, 64, 128, 104, 48, 50, R.moe(4, 4, 24, 2, 2), 500.0, 0.1)], eps=3e-5, scale=7.0)
# Experts that are chosen: groups, one and several kept, one expert per group.
ROUTED = R.config(64, 131, [R.latent(4, 24, 16, 16, 32, 32, 20, R.moe(12, 3, 24, 3, 2)), R.mlstm_layer(2, 16, 24, 12.0, R.moe(10, 2, 40)),
                            R.latent(2, 16, 8, 24, 24, 16, 9, R.moe(8, 1, 32, 8, 3), 100.0, 0.3)], scale=2.5)
# Sizes the tensor-core kernels do not take (not multiples of 8, odd widths), a single head, windows of one and two positions.
ODD = R.config(70, 97, [R.mlstm_layer(1, 10, 14, 5.0, R.moe(2, 2, 13)), R.latent(3, 20, 6, 12, 33, 21, 9, R.moe(3, 3, 51), 500.0, 0.3),
                        R.latent(1, 9, 4, 11, 18, 7, 1), R.mlstm_layer(3, 7, 5, 15.0), R.latent(2, 12, 2, 20, 20, 15, 2)])
SMALL = R.config(64, 97, [R.mlstm_layer(2, 16, 24, 15.0), R.latent(4, 24, 8, 16, 32, 40, 40, R.moe(3, 3, 48)), R.mlstm_layer(1, 40, 64, 15.0)], scale=8.0)
LIMIT = {torch.float32: 3e-4, torch.bfloat16: 0.06}


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
    s = scale or float(want.abs().max())
    limit = limit or (2e-5 if dt == torch.float32 else 1.2e-2)
    assert got.shape == want.shape and float((got - want).abs().max()) <= limit * s, float((got - want).abs().max()) / s


# ---------------------------------------------------------------------------------------------- configuration
def test_config_keeps_every_layer_and_round_trips():
    cfg = ModelConfig.from_hf_dict(MIXED)
    assert cfg.model_type == "lenitar" and cfg.num_hidden_layers == 5 and cfg.is_hybrid and cfg.vocab_size == 211 and cfg.embedding_scale == 7.0
    assert [cfg.layer_has_kv(i) for i in range(5)] == [True, False, True, False, True]
    assert cfg.layer_kv_dims(0) == (1, 48, 0) and cfg.layer_kv_dims(4) == (1, 168, 0)
    assert cfg.layer_state_shape(0) is None and cfg.layer_state_shape(1) == (2 * (24 * 40 + 24 + 1) + 2,) and cfg.layer_state_shape(3)[0] >= 3 * (16 * 137 + 1)
    assert cfg.mixers[0].window == 37 and cfg.mixers[2].scale == 0.15 and cfg.mixers[2].moe is None and cfg.mixers[1].moe.topk_group == 2
    assert ModelConfig.from_hf_dict(cfg.to_hf_dict()).mixers == cfg.mixers
    for change in ({"type": "attention"}, {"mlp": {"kind": "dense", "ff": 4}}, {"mlp": R.moe(10, 2, 8, 3, 1)}, {"mlp": R.moe(8, 5, 8, 4, 2)}):
        wrong = json.loads(json.dumps(MIXED))
        wrong["layers"][0].update(change)
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(wrong)


def test_cache_rows_hold_the_latent_and_states_go_by_layer():
    eng = engine_for(MIXED, R.weights(MIXED), "cpu", torch.float32, state_slots=3)
    assert len(eng.kv.pools) == 3 and eng.kv.layer(2)[0].shape[1:] == (1, 16, 96) and eng.kv.layer(2)[1].numel() == 0
    assert eng.kv.layer_state[1].shape == (3, 2 * (24 * 41 + 1) + 2) and 0 not in eng.kv.layer_state
    S, n, m = ops.mlstm_state_views(eng.kv.layer_state[1][0], 2, 24, 40)
    assert S.shape == (2, 24, 40) and n.shape == (2, 24) and m.shape == (2,)


# ---------------------------------------------------------------------------------------------- mechanisms
@both
@pytest.mark.parametrize("width", [33, 96, 1000, 1028, 2500, 9000])
def test_stream_and_norm_of_the_sum(dev, dt, width):
    M, k = 5, 3
    x = (rand(M, width, seed=1) * 3 + 0.7).float()
    y, rows = rand(M, width, seed=2), rand(9, width, seed=3)
    pos = torch.tensor([0, 8, -1, 3, 3, 1, 7, -1, -1, 2, 4, 5, 6, 0, 8], dtype=torch.int32)
    w = torch.rand(M, k, generator=torch.Generator().manual_seed(4))
    g, b = torch.rand(width) + 0.5, torch.randn(width)
    add = torch.stack([sum((float(w[t, s]) * rows[int(pos[t * k + s])] for s in range(k) if pos[t * k + s] >= 0), torch.zeros(width, dtype=torch.float64))
                       for t in range(M)])
    routed = moe_ops.RoutedRows(rows.to(dev, dt), pos.to(dev), w.to(dev))
    for yy, rr in ((y, routed), (y, None), (None, routed), (None, None)):
        want = x.double() + (y if yy is not None else 0) + (add if rr is not None else 0)
        s, act = ops.residual_norm(x.to(dev), None if yy is None else yy.to(dev, dt), rr, g.to(dev), b.to(dev), 1e-4, dt)
        close(s, want, torch.float32)
        close(act, R.layer_norm(want, g, b, 1e-4), dt)
        s, act = ops.residual_norm(x.to(dev), None if yy is None else yy.to(dev, dt), rr, g.to(dev), None, 1e-4, dt, center=False)
        close(act, R.rms(want, 1e-4) * g.double(), dt)
        s, act = ops.residual_norm(x.to(dev), None if yy is None else yy.to(dev, dt), rr, act_dtype=dt)
        assert act is None
        close(s, want, torch.float32)
    table, ids = rand(11, width, seed=5), torch.tensor([3, 0, 10], dtype=torch.int32)
    s, act = ops.embedding_stream(ids.to(dev), table.to(dev, dt), scale=3.7, want_act=False)
    assert act is None or dt == torch.float32
    close(s, table[ids.long()] * 3.7, torch.float32)


@both
@pytest.mark.parametrize("E,top,groups,keep", [(10, 3, 2, 1), (12, 3, 3, 2), (8, 2, 1, 1), (8, 3, 8, 3), (64, 6, 8, 4), (256, 8, 8, 4), (30, 4, 3, 3), (512, 32, 32, 4)])
def test_routing_by_groups(dev, dt, E, top, groups, keep):
    T = 70
    z = rand(T, E, seed=1) * 2
    z[0] = torch.linspace(-3, 3, E)                                       # the best experts sit in one group
    z[1] = -z[0]
    z[2] = -5.0
    z[2, ::E // groups] = 4.0 - torch.arange(groups).double() * 1e-3                     # one loud expert per group
    z = z + torch.arange(E) * 1e-6
    wide = torch.full((T, E + 5), 9.0)
    wide[:, 5:] = z.float()
    wide = wide.to(dev)
    ids, w = moe_ops.route(wide[:, 5:], top, "sigmoid", False, 1.0, None, groups, keep)
    for t in range(T):
        want = R.route(z[t].float().double(), top, groups, keep)
        got = dict(zip(ids[t].tolist(), w[t].tolist()))
        assert set(got) == {e for e, _ in want}, t
        for e, s in want:
            assert abs(got[e] - float(s)) < 2e-6
    if dev == "cuda" and dt == torch.bfloat16:
        x = rand(T, 64, seed=2).to(dev, dt)
        ids2, w2, plan, xp = moe_ops.route_plan_gather(wide[:60, 5:], x[:60], top, "sigmoid", False, 1.0, None, 0, E, groups, keep)
        assert torch.equal(ids2, ids[:60]) and torch.equal(w2, w[:60])


@both
@pytest.mark.parametrize("T,W,ff,E,top", [(1, 64, 24, 4, 2), (40, 96, 40, 6, 3), (200, 64, 96, 5, 2), (130, 70, 51, 3, 1), (33, 40, 13, 7, 7), (700, 64, 64, 3, 2), (450, 72, 128, 2, 1)])
def test_experts_of_every_route(dev, dt, T, W, ff, E, top):
    x, gu, dn = rand(T, W, seed=1), rand(E, 2 * ff, W, seed=2) / 8, rand(E, W, ff, seed=3) / 8
    gu, dn = gu.to(torch.bfloat16).double(), dn.to(torch.bfloat16).double()
    ids = torch.stack([torch.randperm(E, generator=torch.Generator().manual_seed(t))[:top] for t in range(T)]).int()
    rows, pos = moe_ops.expert_rows(x.to(dev, dt), ids.to(dev), gu.to(dev, dt), dn.to(dev, dt))
    got = rows[pos.long()].double().cpu().view(T, top, W)
    for t in range(0, T, 1 + T // 150):
        for s in range(top):
            e = int(ids[t, s])
            w = {"gate": gu[e, :ff], "up": gu[e, ff:], "down": dn[e]}
            want = R.expert("", w, x[t])
            assert float((got[t, s] - want).abs().max()) <= (2e-5 if dt == torch.float32 else 2e-2) * float(want.abs().max()) + 1e-6


@both
@pytest.mark.parametrize("q_rank,rank,rot", [(24, 40, 8), (7, 18, 4), (512, 256, 64), (96, 33, 2)])
def test_latent_preparation(dev, dt, q_rank, rank, rot):
    M, eps = 7, 1e-3
    positions = torch.tensor([0, 1, 15, 16, 17, 1000, 5])
    slots = torch.tensor([17, 40, 2 * 16 + 15, 3 * 16, 5, -1, 63])
    x = rand(M, q_rank + rank + rot + 3, seed=1) * 2
    qw, kw = rand(q_rank, seed=2) + 1, rand(rank, seed=3) + 1
    inv = torch.tensor([300.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float32)
    cache = torch.zeros(4, 1, 16, rank + rot, device=dev, dtype=dt)
    cq = ops.latent_prepare(x.to(dev, dt), q_rank, rank, rot, qw.float().to(dev), kw.float().to(dev), eps, positions.int().to(dev), slots.to(dev),
                            inv.to(dev), cache)
    close(cq, R.rms(x[:, :q_rank], eps) * qw, dt)
    c = R.rms(x[:, q_rank:q_rank + rank], eps) * kw
    a = (positions.double()[:, None] * inv.double()[None])
    u, v = x[:, q_rank + rank:q_rank + rank + rot // 2], x[:, q_rank + rank + rot // 2:q_rank + rank + rot]
    kr = torch.cat((u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin()), -1)
    for m, s in enumerate(slots.tolist()):
        if s >= 0:
            close(cache[s // 16, 0, s % 16, :rank], c[m], dt)
            close(cache[s // 16, 0, s % 16, rank:], kr[m], dt, limit=5e-4 if dt == torch.float32 else None)
    filled = {s for s in slots.tolist() if s >= 0}
    assert all(s in filled or not cache[s // 16, 0, s % 16].any() for s in range(64))


@pytest.mark.gpu
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("M,H,N,K,rot", [(1, 3, 40, 24, 8), (17, 2, 64, 128, 64), (40, 4, 136, 72, 16), (130, 3, 24, 512, 0), (5, 2, 33, 18, 4)])
def test_one_matrix_per_head(dt, M, H, N, K, rot):
    dev = "cuda"
    x, w = rand(M, H, K + rot, seed=1), rand(H, N, K, seed=2) / 4
    w = w.to(torch.bfloat16).double()
    want = torch.einsum("mhk,hnk->mhn", x[..., :K], w)
    pos = torch.arange(M) * 7
    inv = torch.tensor([50.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float32)
    a = (pos.double()[:, None] * inv.double()[None])[:, None, :]
    u, v = x[..., K:K + rot // 2], x[..., K + rot // 2:]
    tail = torch.cat((u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin()), -1)
    out = torch.zeros(M, H, N + rot, device=dev, dtype=dt)
    ops.head_linear(x.to(dev, dt), w.to(dev, dt), out, rot=rot, positions=pos.int().to(dev), inv_freq=inv.to(dev))
    close(out[..., :N], want, dt)
    if rot:
        close(out[..., N:], tail, dt, limit=5e-4 if dt == torch.float32 else None)
    rows = torch.tensor([m for m in range(M) if m % 3 != 1], dtype=torch.int32)
    part = torch.zeros(len(rows), H, N + rot, device=dev, dtype=dt)
    ops.head_linear(x.to(dev, dt), w.to(dev, dt), part, in_rows=rows.to(dev), rot=rot, positions=pos.int().to(dev), inv_freq=inv.to(dev))
    assert torch.equal(part, out[rows.long().to(dev)])
    gate = rand(M, H * N + 8, seed=3)
    back = torch.full((M, H, N), 5.0, device=dev, dtype=dt)
    ops.head_linear(x[rows.long(), :, :K].contiguous().to(dev, dt), w.to(dev, dt), back, gate=gate.to(dev, dt)[:, 8:], out_rows=rows.to(dev))
    gated = want * R.sigmoid(gate[:, 8:]).view(M, H, N)
    close(back[rows.long().to(dev)], gated[rows.long()], dt)
    assert all(bool((back[m] == 5.0).all()) for m in range(M) if m % 3 == 1)


def prompt_batch(portions, tables, dev):
    """ForwardBatch of prompt portions [(first new position, new tokens)] over the given page lists."""
    cu = torch.tensor([0] + [n for _, n in portions]).cumsum(0)
    width = max(len(t) for t in tables)
    return ForwardBatch(token_ids=None, positions=torch.cat([torch.arange(a, a + n) for a, n in portions]).int().to(dev), slots=None,
                        block_table=torch.tensor([t + [0] * (width - len(t)) for t in tables], dtype=torch.int32, device=dev),
                        seq_lens=torch.tensor([a + n for a, n in portions], dtype=torch.int32, device=dev), is_prefill=True,
                        cu_q=cu.int().to(dev), max_q_len=max(n for _, n in portions), portions=list(portions))


def decode_batch(lens, tables, dev, most):
    width = max(len(t) for t in tables)
    return ForwardBatch(token_ids=None, positions=torch.tensor([n - 1 for n in lens], dtype=torch.int32, device=dev), slots=None,
                        block_table=torch.tensor([t + [0] * (width - len(t)) for t in tables], dtype=torch.int32, device=dev),
                        seq_lens=torch.tensor(lens, dtype=torch.int32, device=dev), is_prefill=False, q_per_seq=1, max_kv_len=most)


ATTENTION = [(4, 40, 24, 88, 112, 78), (3, 16, 8, 24, 40, 37), (2, 128, 64, 128, 256, 100), (5, 64, 64, 64, 128, 16), (1, 72, 16, 40, 512, 128),
             (20, 24, 16, 32, 64, 200), (2, 100, 24, 8, 48, 1), (3, 20, 6, 12, 33, 9), (1, 9, 4, 11, 18, 2), (40, 16, 8, 16, 384, 0)]


@both
@pytest.mark.parametrize("H,dim,rot,vdim,rank,window", ATTENTION)
def test_latent_attention_sees_its_window_and_the_sink(dev, dt, H, dim, rot, vdim, rank, window, monkeypatch):
    """Keys around window edges, page borders and the first tokens are made to stand out: one just inside or just outside a query's
    window decides the whole row."""
    T, base, scale = 330, 100.0, 1.0
    g = torch.Generator().manual_seed(1)
    uk, uv = rand(H, dim, rank, seed=2) / math.sqrt(rank), rand(H, vdim, rank, seed=3) / math.sqrt(rank)
    uk, uv = uk.to(torch.bfloat16).double(), uv.to(torch.bfloat16).double()
    c, kr = rand(T, rank, seed=4), rand(T, rot, seed=5) * 0.3
    edges = sorted({0, 1, 2, 15, 16, 17, 150, 151, T - 1, T - 2} | {p for p in range(0, T, 37)})
    loud = torch.randn(rank, generator=g).double()                       # every head's queries look for the keys of this latent
    for n, p in enumerate(edges):
        c[p] = c[p] * 0.5 + loud * (1.0 + 0.1 * (n % 5))
    c, kr = c.to(torch.bfloat16).double(), kr.to(torch.bfloat16).double()
    keys = uk @ loud
    qn = rand(T, H, dim, seed=6) * 0.2 + keys * (5.0 / keys.square().sum(-1, keepdim=True))
    qr0 = rand(T, H, rot, seed=7) * 0.3
    q = torch.cat((qn, qr0), -1).to(torch.bfloat16).double()
    inv = torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float32)
    qr = R.rotate(q[..., dim:], torch.arange(T), base, rot)
    sink = torch.linspace(6.0, 1.0, H).float()
    gate = rand(T, H * vdim + 8, seed=8)
    size = window or 10 ** 6

    def oracle(size, sink):
        o = R.latent_heads(q[..., :dim], qr, c, kr, uk, uv, sink.double(), scale, R.window_mask(T, size))
        return o.reshape(T, -1) * R.sigmoid(gate[:, 8:])

    want = oracle(size, sink)
    top = float(want.abs().max())
    if window:
        assert float((oracle(size + 1, sink) - want).abs().max()) > 0.1 * top        # an edge that is off by one would show
        assert window < 3 or float((oracle(size - 1, sink) - want).abs().max()) > 0.1 * top
    assert float((oracle(size, sink - 100) - want).abs().max()) > 0.1 * top
    pages = [(i * 8) % 21 + 1 for i in range(21)]
    cache = torch.full((23, 1, 16, rank + rot), 3.0, device=dev, dtype=dt)
    for t in range(T):
        cache[pages[t // 16], 0, t % 16] = torch.cat((c[t], kr[t])).to(dev, dt)
    kv_up = torch.cat((uk.reshape(-1, rank), uv.reshape(-1, rank))).to(dev, dt)
    ukt, uvd = uk.transpose(1, 2).contiguous().to(dev, dt), uv.to(dev, dt)
    limit = 2e-5 if dt == torch.float32 else 2.5e-2

    def run(rows, batch):
        y = ops.latent_attention(q[rows].reshape(len(rows), -1).to(dev, dt).contiguous(), cache, batch, ukt, uvd, kv_up,
                                 gate[rows].to(dev, dt)[:, 8:], sink.to(dev), inv.to(dev), H, dim, rot, scale, window)
        assert float((y.double().cpu() - want[rows]).abs().max()) <= limit * top, (batch.portions, batch.seq_lens)

    spans = [(0, T), (0, 130), (33, 35), (95, 200), (199, 330), (328, 330), (0, 2)]
    for cost in (1e9, 0.0, None):                                        # always expanded where it can be, never, by arithmetic
        if cost is not None:
            monkeypatch.setattr(latent_ops, "ABSORBED_COST", cost)
        else:
            monkeypatch.undo()
        for a, b in spans:
            run(list(range(a, b)), prompt_batch([(a, b - a)], [pages], dev))
    mixed = [(0, 140), (200, 1), (70, 2), (299, 31), (12, 9), (329, 1)]
    run([p for a, n in mixed for p in range(a, a + n)], prompt_batch(mixed, [pages] * len(mixed), dev))
    at = sorted({p for e in edges for p in (e, e + 1, e + size - 1, e + size) if p < T} | {0, 1, 200})
    for most in (0, T, 4096):                                            # how far a step may see chooses the split of the keys
        run(at, decode_batch([p + 1 for p in at], [pages] * len(at), dev, most))
    run(at[-2:], decode_batch([p + 1 for p in at[-2:]], [pages] * 2, dev, T))


def ragged(rows, starts, pages, dev):
    """ForwardBatch of portions: sequence i brings rows[i] tokens from position starts[i]; its first page is pages[i]."""
    cu = torch.tensor([0] + rows).cumsum(0)
    slots = torch.cat([torch.arange(r) + pages[i] * 16 for i, r in enumerate(rows)])
    return ForwardBatch(token_ids=torch.zeros(int(cu[-1]), dtype=torch.int32, device=dev), positions=torch.zeros(int(cu[-1]), dtype=torch.int32),
                        slots=slots.to(dev), block_table=torch.tensor([[p, 0] for p in pages], dtype=torch.int32, device=dev),
                        seq_lens=torch.tensor([s + r for s, r in zip(starts, rows)], dtype=torch.int32, device=dev),
                        is_prefill=True, cu_q=cu.int().to(dev), max_q_len=max(rows))


def mlstm_inputs(T, H, D, V, seed, kind):
    """Projections and gate pre-activations. "plain"; "keep": nothing is forgotten and the inputs close after the first tokens, so what
    they wrote still counts; "loud": input gates up to the cap, where the small constant of the normaliser matters; "swing": both
    gates change abruptly."""
    x = rand(T, 2 * H * D + 2 * H * V, seed=seed)
    z = rand(T, 2 * H, seed=seed + 1) * 2
    z[:, H:] += 2
    if kind == "keep":
        z[:, H:] = 14.0
        z[:, :H] -= 4.0
        z[:3, :H] = 3.0
    elif kind == "loud":
        z[:, :H] = z[:, :H] * 4 + 20.0
    elif kind == "swing":
        z[:, H:] = torch.where(torch.arange(T)[:, None] % 23 == 5, -30.0, 6.0)
        z[:, :H] = torch.where(torch.arange(T)[:, None] % 17 == 3, 12.0, -6.0)
    return x, z.float().double(), rand(H * V, seed=seed + 2) * 0.3 + 1


def mlstm_reference(x, z, nw, H, D, V, cap, eps, state):
    T, qk, vw = x.shape[0], H * D, H * V
    i, f = R.mlstm_gates(z[:, :H], z[:, H:], cap)
    o, state = R.mlstm_scan((x[:, :qk] * D ** -0.5).view(T, H, D), x[:, qk:2 * qk].view(T, H, D), x[:, 2 * qk:2 * qk + vw].view(T, H, V), i, f, state)
    return R.rms(o, eps).reshape(T, vw) * nw * R.sigmoid(x[:, 2 * qk + vw:]), state


PORTIONS = [[300], [1] * 12 + [40, 2, 2, 100, 64, 65, 15], [64, 128, 16, 8, 9, 75]]


@both
@pytest.mark.parametrize("portions", PORTIONS)
@pytest.mark.parametrize("H,D,V,cap,kind", [(3, 24, 40, 9.0, "plain"), (2, 64, 128, 15.0, "keep"), (1, 128, 256, 15.0, "loud"), (2, 16, 64, 15.0, "swing"),
                                            (1, 256, 392, 12.0, "plain"), (2, 40, 56, 15.0, "loud"), (1, 20, 30, 2.0, "swing"), (3, 7, 5, 15.0, "keep")])
def test_matrix_memory(dev, dt, H, D, V, cap, kind, portions):
    T = 300
    x, z, nw = mlstm_inputs(T, H, D, V, 7, kind)
    want, (S, n, m) = mlstm_reference(x, z, nw, H, D, V, cap, 1e-5, R.mlstm_start(H, D, V))
    size = -(-H * (D * V + D + 1) // 4) * 4
    state = torch.zeros(2, size, device=dev)
    p2s = torch.tensor([0, 1, 0], dtype=torch.int32, device=dev)
    outs, at, i = [], 0, 0
    while at < T:
        k = min(portions[min(i, len(portions) - 1)], T - at)
        outs.append(ops.mlstm(x[at:at + k].contiguous().to(dev, dt), z[at:at + k].float().contiguous().to(dev), nw.float().to(dev), state, H, D, V, cap,
                              1e-5, ragged([k], [at], [1], dev), p2s))
        at, i = at + k, i + 1
    close(torch.cat(outs), want, dt, limit=5e-5 if dt == torch.float32 else None)
    gS, gn, gm = ops.mlstm_state_views(state[1], H, D, V)
    for got, exp in ((gS, S), (gn, n), (gm, m)):                      # the state is fp32 in both
        close(got, exp, torch.float32, scale=float(exp.abs().max()) * (5 if dt == torch.float32 else 10) + 1e-9)
    assert not state[0].any()


@both
def test_matrix_memory_of_a_ragged_batch_and_idle_rows(dev, dt):
    """Portions of unequal length side by side give what each gives alone; a row without a cache slot keeps its state."""
    H, D, V, cap = 2, 32, 48, 11.0
    rows, pages = [70, 1, 130, 2, 64, 17], [3, 1, 5, 2, 4, 6]
    x, z, nw = mlstm_inputs(sum(rows), H, D, V, 3, "plain")
    f = lambda t: t.float().contiguous().to(dev)                                       # noqa: E731
    size = H * (D * V + D + 1) + 2
    st = f(rand(6, size, seed=5))
    st0 = st.clone()
    p2s = torch.tensor([0, 4, 1, 0, 3, 2, 5], dtype=torch.int32, device=dev)
    step = lambda a, b, s, bt: ops.mlstm(x[a:b].contiguous().to(dev, dt), f(z[a:b]), f(nw), s, H, D, V, cap, 1e-5, bt, p2s)     # noqa: E731
    batch = ragged(rows, [9] * 6, pages, dev)
    got, at = step(0, sum(rows), st, batch), 0
    for i, n in enumerate(rows):
        alone = st0.clone()
        close(got[at:at + n], step(at, at + n, alone, ragged([n], [9], [pages[i]], dev)).double().cpu(), dt)
        slot = int(p2s[pages[i]])
        close(st[slot], alone[slot].double().cpu(), torch.float32)
        at += n
    idle = ForwardBatch(token_ids=None, positions=None, slots=torch.tensor([5, -1, 9, -1, 3, 7], device=dev), block_table=batch.block_table,
                        seq_lens=batch.seq_lens, is_prefill=False, q_per_seq=1)
    st = st0.clone()
    step(0, 6, st, idle)
    for i in range(6):
        slot = int(p2s[pages[i]])
        assert torch.equal(st[slot], st0[slot]) == (i in (1, 3))


# ---------------------------------------------------------------------------------------------- whole models
def agrees(got, want, dt, exact=True):
    """Every position within rounding. ``exact`` False: where rounding may change an expert, most positions in bf16."""
    e = R.errors(got, want)
    worst = e.max() if exact or dt == torch.float32 else e.quantile(0.8)
    assert float(worst) < LIMIT[dt], (float(e.max()), int(e.argmax()), float(e.quantile(0.8)))


@both
@pytest.mark.parametrize("cfg,exact", [(MIXED, True), (ODD, True), (ROUTED, False)], ids=["mixed", "odd", "routed"])
def test_prompt_portions_and_decoding_agree_with_the_restatement(dev, dt, cfg, exact):
    w = R.weights(cfg, seed=1)
    tokens = prompt(150, cfg["vocab"], 2)
    want = R.forward(cfg, w, tokens)
    eng = engine_for(cfg, w, dev, dt, max_seq_len=160, num_pages=11, state_slots=1)      # room for one: every run reuses it
    for sizes in ([150], [100, 1], [2, 3, 2, 17, 64], [37, 20, 43, 50], [1]):
        seq = eng.open_sequence()
        agrees(feed(eng, seq, tokens, sizes), want, dt, exact)
        eng.release(seq)


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
    for layer, change in ((0, {"mask": {"size": 38}}), (0, {"mask": {"size": 36}}), (2, {"mask": {"size": 17}}), (2, {"scale": 0.3}),
                          (4, {"rot": {"dims": 64, "base": 50.0}}), (1, {"gate_cap": 4.0})):
        other = json.loads(json.dumps(MIXED))
        other["layers"][layer]["mixer"].update(change)
        assert R.error(got, R.forward(other, w, tokens)) > 2 * LIMIT[dt], (layer, change)
    for name, factor in (("l0.mix.sink", -9.0), ("l1.mix.i", 0.0), ("l1.mix.f", 0.0), ("l0.norm1.b", 0.0), ("final.norm.b", 0.0)):
        other = dict(w, **{name: w[name] * factor})
        assert R.error(got, R.forward(MIXED, other, tokens)) > 2 * LIMIT[dt], name


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
def test_long_decoding_across_windows(dev, dt):
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

    w = R.weights(MIXED, seed=10)
    mc = save(tmp_path / "m", MIXED, w)
    report = inspect_artifact(tmp_path / "m")
    assert report.is_loadable and report.model_type == "lenitar"
    prof = estimate_runtime_state(mc)
    assert prof.kv_bytes_per_token == 2 * (48 + 96 + 168) and prof.state_bytes_per_sequence == 4 * (mc.layer_state_shape(1)[0] + mc.layer_state_shape(3)[0])
    assert abs(prof.expert_bytes - 2 * 3 * 96 * (3 * 40 + 2 * 72 + 4 * 24)) <= 8
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


@both
def test_observer_sees_outputs_and_routing_and_may_replace_them(dev, dt):
    from eredu_b200.runtime.inspection import ActivationObserver

    class Watch(ActivationObserver):
        def __init__(self):
            self.routing, self.outputs = [], []

        def observe(self, name, value):
            self.outputs.append(name)

        def intervene(self, name, value):
            return value * 0 if name == "model.layers.1.output" else None

        def observe_moe_routing(self, o):
            self.routing.append(o)

    w = R.weights(MIXED, seed=12)
    tokens = prompt(20, MIXED["vocab"], 5)
    eng = engine_for(MIXED, w, dev, dt)
    plain = feed(eng, eng.open_sequence(), tokens, [20])
    eng.model.observer = watch = Watch()
    changed = feed(eng, eng.open_sequence(), tokens, [20])
    assert [o.num_experts for o in watch.routing] == [3, 2, 4] and watch.routing[0].selected_experts.shape == (20, 3)
    assert "model.layers.4.output" in watch.outputs and R.error(changed, plain.double().cpu()) > 0.1
    watch.intervene = lambda name, value: None
    agrees(feed(eng, eng.open_sequence(), tokens, [20]), R.forward(MIXED, w, tokens), dt)


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
    assert 0 < t["generated_tokens"] <= 6 and t["plan"]["model_type"] == "lenitar" and "TTFT" in capsys.readouterr().err


def test_random_models_of_a_configuration():
    from eredu_b200.models.llama import build_random, random_state

    mc = ModelConfig.from_hf_dict(SMALL)
    sd = random_state(mc, seed=3)
    a, b = build_from_tensors(mc, sd.__getitem__, sd.__contains__, "cpu", torch.float32), build_random(mc, "cpu", torch.float32, seed=3)
    assert torch.equal(a.layers[1].moe.w_down, b.layers[1].moe.w_down) and a.weight_bytes() > 0
    assert Engine(a, max_batch=1, max_seq_len=64).generate([[1, 2, 3]], SamplingParams(temperature=0.0), 4) == \
        Engine(b, max_batch=1, max_seq_len=64).generate([[1, 2, 3]], SamplingParams(temperature=0.0), 4)
