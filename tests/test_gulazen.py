"""Gulazen: every mechanism alone and whole models against the plain restatement in gulazen_reference.py - prompts, decoding, portions,
unequal batches, reused pages and slots, edges of windows and of the kept first tokens, greedy generation through the engine and the
server."""
import json
import math

import pytest
import torch

import gulazen_reference as R
from eredu_b200 import ops
from eredu_b200.models.config import ModelConfig
from eredu_b200.models.llama import ForwardBatch, build_from_tensors
from eredu_b200.ops import SamplingParams
from eredu_b200.runtime.engine import Engine

CASES = [pytest.param("cpu", torch.float32, id="cpu-fp32"), pytest.param("cuda", torch.float32, marks=pytest.mark.gpu, id="gpu-fp32"),
         pytest.param("cuda", torch.bfloat16, marks=pytest.mark.gpu, id="gpu-bf16")]
both = pytest.mark.parametrize("dev,dt", CASES)

# Sizes that are unequal where they can be; windows and kept tokens that end inside pages and on them; every kind of feed-forward and none.
MIXED = R.config(96, 211, [R.attention_layer(6, 2, 24, 40, 37, 5, R.dense_ff(88), scale=0.3, cap=7.0),
                           R.attention_layer(4, 4, 64, 16, 16, 16, R.expert_ff(7, 3, 24, 56), scale=0.12, cap=30.0),
                           R.attention_layer(2, 1, 72, 128, 50, 33, None, scale=0.1, cap=12.0),
                           R.attention_layer(12, 4, 16, 24, 21, 0, R.expert_ff(4, 1, 40), scale=0.25, cap=15.0),
                           R.attention_layer(3, 3, 128, 8, 33, 1, R.dense_ff(40), scale=0.09, cap=50.0)], taps=4, eps=3e-5)
# Sizes the tensor-core kernels do not take (not multiples of 8, odd widths), one head, one expert, one tap, windows of one.
ODD = R.config(71, 97, [R.attention_layer(3, 1, 9, 13, 7, 2, R.dense_ff(51), scale=0.4, cap=9.0),
                        R.attention_layer(1, 1, 20, 5, 1, 3, R.expert_ff(3, 3, 11, 13), scale=0.3),
                        R.attention_layer(10, 5, 12, 7, 20, 17, R.expert_ff(1, 1, 20), scale=0.3)], taps=1)
SMALL = R.config(64, 97, [R.attention_layer(4, 2, 32, 24, 40, 9, R.dense_ff(72)), R.attention_layer(2, 2, 40, 32, 24, 20, R.expert_ff(6, 2, 32, 48))], taps=2)
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
    assert cfg.model_type == "gulazen" and cfg.num_hidden_layers == 5 and cfg.is_hybrid and cfg.vocab_size == 211 and cfg.tie_word_embeddings
    assert all(cfg.layer_has_kv(i) for i in range(5)) and cfg.layer_kv_dims(0) == (2, 24, 40) and cfg.layer_kv_dims(4) == (3, 128, 8)
    assert cfg.layer_state_shape(2) == (3 * 96,)
    a, b = cfg.mixers[0], cfg.mixers[1]
    assert (a.window, a.keep_first, a.softcap, a.scale, a.ff, a.moe) == (37, 5, 7.0, 0.3, 88, None)
    assert (b.moe.num_experts, b.moe.num_experts_per_tok, b.moe.moe_intermediate_size, b.moe.shared_ff) == (7, 3, 24, 56)
    assert cfg.mixers[2].ff == 0 and cfg.mixers[2].moe is None and cfg.mixers[3].moe.shared_ff == 0
    assert ModelConfig.from_hf_dict(cfg.to_hf_dict()).mixers == cfg.mixers
    assert not ModelConfig.from_hf_dict(ODD).is_hybrid                       # one tap keeps no history
    for change in ({"type": "gla"}, {"mlp": {"kind": "sparse"}}, {"mlp": R.expert_ff(4, 5, 8)}):
        wrong = json.loads(json.dumps(MIXED))
        wrong["layers"][0].update(change)
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(wrong)
    for change in ({"kv_heads": 4}, {"mask": {"size": 0, "keep_first": 4}}, {"mask": {"size": 9, "keep_first": -1}}, {"softcap": -1.0}):
        wrong = json.loads(json.dumps(MIXED))
        wrong["layers"][0]["mixer"].update(change)
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(wrong)


# ---------------------------------------------------------------------------------------------- mechanisms
@both
@pytest.mark.parametrize("width", [33, 96, 256, 1001, 4096])
def test_embedding_with_position_vectors(dev, dt, width):
    table = rand(50, width, seed=1)
    ids, pos = torch.tensor([3, 49, 0, 7, 7, 12]), torch.tensor([0, 1, 2, 500, 501, 9000])
    inv = torch.tensor([10000.0 ** (-2.0 * i / width) for i in range((width + 1) // 2)], dtype=torch.float64).float()
    x, act = ops.embedding_stream(ids.int().to(dev), table.to(dev, dt), positions=pos.int().to(dev), inv_freq=inv.to(dev))
    want = table[ids] + R.position_vectors(pos, width, torch.float64)
    assert x.dtype == torch.float32
    close(x[:5], want[:5], torch.float32, scale=1.0, limit=1e-4)                        # angles in fp32
    close(x, want, torch.float32, scale=1.0, limit=2e-3)
    close(act, want, dt, limit=2e-3 if dt == torch.float32 else None)


@both
@pytest.mark.parametrize("width", [33, 96, 1000, 2500, 8192, 9000])
def test_norm_behind_a_sublayer_and_its_expert_rows(dev, dt, width):
    M, k, eps = 5, 3, 1e-4
    x, y, rows = rand(M, width, seed=1).float(), rand(M, width, seed=2) * 0.02, rand(M * k, width, seed=3) * 0.03
    y, rows = (t.to(torch.bfloat16).double() for t in (y, rows))
    weight, w = rand(width, seed=4) * 0.2 + 1, torch.rand(M, k, generator=torch.Generator().manual_seed(5)).double()
    order = torch.randperm(M * k, generator=torch.Generator().manual_seed(6))
    stored = torch.empty_like(rows)
    stored[order] = rows
    routed = ops_rows(stored.to(dev, dt), order.int().to(dev), w.float().to(dev))
    summed = (rows.view(M, k, width) * w[..., None]).sum(1)
    on = lambda t: None if t is None else t.to(dev, dt)                                 # noqa: E731
    for own, r in ((y, None), (y, routed), (None, routed)):
        s = (0 if own is None else own) + (0 if r is None else summed)
        want = x.double() + R.unit_rms(s, eps) * weight
        for act in (True, False):
            out, copy = ops.rms_residual(on(own), weight.float().to(dev), eps, residual=x.to(dev), act_dtype=dt, routed=r, want_act=act)
            close(out, want, torch.float32)
            assert (copy is None) != act
            if act:
                close(copy, want, dt)


def ops_rows(rows, pos, weights):
    from eredu_b200.ops.moe import RoutedRows

    return RoutedRows(rows, pos, weights)


@both
@pytest.mark.parametrize("above,below", [(0.3, 0.9), (2.0, 0.5), (1e-3, 3.0)])
@pytest.mark.parametrize("M,K,N", [(1, 64, 40), (3, 70, 51), (40, 96, 128), (130, 64, 72), (300, 128, 64), (700, 64, 200)])
def test_xielu_of_a_projection(dev, dt, M, K, N, above, below):
    """Small and large pre-activations of both signs."""
    inv = lambda t: math.log(math.expm1(t)) if t > 0 else -math.inf                      # noqa: E731
    x, w = rand(M, K, seed=1), (rand(N, K, seed=2) / 8).to(torch.bfloat16).double()
    x[::3] = (x[::3] * 0.01).to(torch.bfloat16).double()
    act = ops.XIELU(above, below)
    z = x @ w.t()
    want = R.xielu(z, torch.tensor(inv(above), dtype=torch.float64), torch.tensor(inv(below - 0.5), dtype=torch.float64))
    got = ops.linear(x.to(dev, dt), w.to(dev, dt), activation=act)
    close(got, want, dt)
    small = torch.arange(M) % 3 == 0
    close(got[small.to(dev)], want[small], dt)
    p, q = 0.7, -0.4
    assert ops.XIELU.from_checkpoint(p, q).above == pytest.approx(math.log1p(math.exp(p))) and ops.XIELU.from_checkpoint(p, q).below == pytest.approx(0.5 + math.log1p(math.exp(q)))


@both
@pytest.mark.parametrize("width,taps", [(96, 2), (100, 3), (256, 4), (33, 3), (2052, 1), (64, 6), (40, 20)])
def test_convolution_of_the_stream(dev, dt, width, taps):
    """One portion, portions of every kind and token by token; in decode steps also behind the norm of the sublayer in front."""
    T = 90
    x, t = rand(T, width, seed=1).float(), rand(taps, width, seed=2) / taps ** 0.5
    want = x.double() + R.causal_conv(x.double(), t.t())
    table = [5, 2, 7, 1, 3, 6]
    p2s = torch.zeros(8, dtype=torch.int32, device=dev)
    p2s[5] = 2
    hist = (taps - 1) * width
    for sizes in ([T], [1], [40, 1, 1, 2, 3, 16, 5, 22], [2, 1, 7, 17, 33, 30]):
        for extra in (0, 5):                                                 # the history may lie in a wider state
            state = torch.zeros(3, hist + extra, device=dev) if taps > 1 else None
            if taps > 1:
                state[:, hist:] = 7.0
                state[0] = 9.0
            at, i, outs = 0, 0, []
            while at < T:
                m = min(sizes[min(i, len(sizes) - 1)], T - at)
                bt = batch_of([(at, m)], [table], dev, prefill=m > 1)
                conv = ops.StreamConv(t.float().contiguous().to(dev), state, bt, p2s)
                part = x[at:at + m].contiguous().to(dev)
                if m == 1 and i % 2:
                    y, wy = rand(1, width, seed=at), rand(width, seed=at + 1).float()
                    res = (part.cpu().double() - R.unit_rms(y, 1e-5) * wy.double()).float()
                    got, act = ops.rms_residual(y.to(dev, dt), wy.to(dev), 1e-5, residual=res.to(dev), act_dtype=dt, conv=conv)
                    close(got, x[at:at + 1], torch.float32)
                else:
                    act = ops.stream_conv(part, conv, dt)
                outs.append(act)
                at, i = at + m, i + 1
            close(torch.cat(outs), want, dt)
            if taps > 1:
                close(state[2, :hist].view(taps - 1, width), x[T - taps + 1:], torch.float32)
                assert bool((state[:, hist:][1:] == 7.0).all()) and bool((state[0] == 9.0).all()) and not state[1, :hist].any()


@both
def test_convolution_of_a_ragged_batch_and_idle_rows(dev, dt):
    W, taps = 72, 4
    rows, starts = [20, 1, 33, 2, 16, 3], [5, 40, 0, 13, 15, 1]
    tables = [[i * 4 + 1 + j for j in range(4)] for i in range(6)]
    x, t = rand(sum(rows), W, seed=1).float().to(dev), rand(taps, W, seed=2).float().to(dev)
    state0 = rand(6, (taps - 1) * W, seed=4).float().to(dev)
    p2s = torch.zeros(25, dtype=torch.int32, device=dev)
    for i, slot in enumerate((4, 1, 0, 3, 2, 5)):
        p2s[tables[i][0]] = slot
    state = state0.clone()
    got = ops.stream_conv(x, ops.StreamConv(t, state, batch_of(list(zip(starts, rows)), tables, dev), p2s), dt)
    at = 0
    for i, m in enumerate(rows):
        alone = state0.clone()
        one = ops.stream_conv(x[at:at + m].contiguous(), ops.StreamConv(t, alone, batch_of([(starts[i], m)], [tables[i]], dev), p2s), dt)
        slot = int(p2s[tables[i][0]])
        assert torch.equal(got[at:at + m], one) and torch.equal(state[slot], alone[slot])
        at += m
    for fused in (False, True):
        bt = batch_of([(s + 1, 1) for s in starts], tables, dev, prefill=False)
        bt.slots = torch.where(torch.tensor([0, 1, 0, 1, 0, 0], device=dev) == 1, -1, bt.slots)
        state = state0.clone()
        conv = ops.StreamConv(t, state, bt, p2s)
        if fused:
            ops.rms_residual(x[:6].to(dt).contiguous(), torch.ones(W, device=dev), 1e-5, residual=x[6:12].contiguous(), act_dtype=dt, conv=conv)
        else:
            ops.stream_conv(x[:6].contiguous(), conv, dt)
        for i in range(6):
            slot = int(p2s[tables[i][0]])
            assert torch.equal(state[slot], state0[slot]) == (i in (1, 3))


@both
def test_router_takes_the_largest_logits_and_weighs_those_alone(dev, dt):
    from eredu_b200.ops import moe

    z = rand(40, 13, seed=1)
    for top in (1, 4, 13):
        idx, want = R.routing(z, top)
        ids, w = moe.route(z.float().to(dev), top, "topk_softmax", False)
        dense = torch.zeros(40, 13, dtype=torch.float64).scatter_(1, ids.long().cpu(), w.double().cpu())
        close(dense, torch.zeros(40, 13, dtype=torch.float64).scatter_(1, idx, want), torch.float32)


ATTENTION = [(6, 2, 24, 40, 37, 5), (4, 4, 64, 16, 16, 16), (2, 1, 72, 128, 50, 33), (12, 4, 16, 24, 21, 0), (3, 3, 128, 8, 33, 1), (16, 4, 128, 128, 100, 7),
             (32, 8, 128, 128, 64, 40), (40, 8, 64, 64, 30, 3), (64, 2, 32, 16, 45, 20), (3, 1, 9, 13, 7, 2), (1, 1, 136, 40, 1, 20), (70, 7, 16, 8, 20, 17), (5, 5, 64, 128, 0, 0),
             (64, 8, 128, 128, 33, 18), (24, 8, 128, 128, 17, 3), (8, 2, 128, 128, 90, 32), (24, 8, 64, 64, 40, 1), (64, 8, 64, 64, 16, 0), (16, 4, 64, 64, 70, 48)]


def loud_inputs(H, G, dk, dv, edges, T):
    """Keys at the given positions stand out for every query, so whether one is seen decides the row."""
    loud = rand(G, dk, seed=9)
    k, v = rand(T, G, dk, seed=1), rand(T, G, dv, seed=2)
    for n, p in enumerate(edges):
        k[p] = k[p] * 0.5 + loud * (1.0 + 0.1 * (n % 5))
    q = rand(T, H, dk, seed=3) * 0.2 / dk ** 0.5 + (loud * (6.0 / loud.square().sum(-1, keepdim=True))).repeat_interleave(H // G, 0)
    exact = lambda t: t.to(torch.bfloat16).double()                                     # noqa: E731
    return exact(q), exact(k), exact(v)


@both
@pytest.mark.parametrize("H,G,dk,dv,window,keep", ATTENTION)
def test_attention_mixes_heads_over_the_window_and_the_first_tokens(dev, dt, H, G, dk, dv, window, keep):
    T, scale, cap = 330, 1.3, 9.0
    edges = sorted({0, 1, 15, 16, 17, 150, 151, T - 1, T - 2, max(0, keep - 1), keep} | set(range(0, T, 37)))
    q, k, v = loud_inputs(H, G, dk, dv, edges, T)
    talk = (torch.eye(H, dtype=torch.float64) * 0.7 + rand(H, H, seed=5) * 0.9 / H ** 0.5).to(torch.bfloat16).double()
    if H > 1:
        talk[0, 1], talk[1, 0] = 0.75, -0.5
    sink = rand(H, seed=6) + 5.0
    size = window or T
    want = R.talking_attention(q, k, v, scale, cap, talk, sink, size, keep)
    top = float(want.abs().max())
    wrong = [dict(talk=talk.t()), dict(talk=torch.eye(H, dtype=torch.float64)), dict(cap=90.0), dict(sink=sink * 0 - 99)]
    wrong = wrong[2:] if H == 1 else wrong
    if window:
        wrong += [dict(size=size + 1)] + ([dict(size=size - 1)] if size > 1 else []) + [dict(keep=keep + 1)] + ([dict(keep=keep - 1)] if keep else [])
    for change in wrong:                                                     # each of these mistakes would show
        other = R.talking_attention(q, k, v, *{**dict(scale=scale, cap=cap, talk=talk, sink=sink, size=size, keep=keep), **change}.values())
        assert float((other - want).abs().max()) > 0.06 * top, change.keys()
    table = [(i * 8) % 21 + 1 for i in range(21)]
    pos = torch.arange(T)
    at_page = torch.tensor(table)[pos // 16]
    kc, vc = (torch.full((23, G, 16, d), 3.0, device=dev, dtype=dt) for d in (dk, dv))
    kc[at_page, :, pos % 16], vc[at_page, :, pos % 16] = k.to(dev, dt), v.to(dev, dt)
    limit = 3e-5 if dt == torch.float32 else 1.5e-2
    talk_d, sink_d = talk.to(dev, dt).contiguous(), sink.float().to(dev)

    def run(portions, prefill=True, most=0):
        rows = [p for a, n in portions for p in range(a, a + n)]
        y = ops.talking_attention(q[rows].contiguous().to(dev, dt), kc, vc, batch_of(portions, [table] * len(portions), dev, prefill, most), talk_d,
                                  scale, cap, sink_d, window, keep)
        err = (y.double().cpu() - want[rows]).abs().flatten(1).max(1).values
        assert float(err.max()) <= limit * top, (portions, prefill, rows[int(err.argmax())], float(err.max()) / top)

    for a, b in [(0, T), (0, 130), (33, 35), (95, 200), (199, 330), (328, 330), (0, 2)]:
        run([(a, b - a)])
    run([(0, 140), (0, 1), (0, 200), (0, 31), (0, 9)])
    run([(200, 1), (202, 2), (200, 130), (299, 31)])
    at = sorted({p for e in edges for p in (e, e + 1, e + size - 1, e + size, e + size + 1) if p < T})
    for most in (0, T, 4096):                                            # how far a step may see chooses the split of the keys
        run([(p, 1) for p in at], prefill=False, most=most)
    run([(p, 1) for p in at[-3:]], prefill=False, most=4096)
    run([(p, 3) for p in at if p + 3 <= T][:7], prefill=False, most=T)
    run([(p, 8) for p in at if p + 8 <= T][-2:], prefill=False, most=T)
    run([(at[-1], 1)], prefill=False, most=T)


@both
def test_scores_are_mixed_in_32_bit(dev, dt):
    """Two heads whose mixture cancels: large scores of which only the difference counts."""
    H, d, T = 2, 32, 64
    k, v = torch.zeros(T, 2, d, dtype=torch.float64), rand(T, 2, d, seed=1)
    q = torch.zeros(1, 2, d, dtype=torch.float64)
    q[..., 0], q[..., 1] = 16.0, 1.0
    k[:, 0, 0] = k[:, 1, 0] = (torch.randn(T, generator=torch.Generator().manual_seed(2)) * 8).to(torch.bfloat16).double()
    k[:, 0, 1] = torch.linspace(-1, 1, T).to(torch.bfloat16).double()
    talk = torch.tensor([[1.0, -1.0], [0.0, 0.0625]], dtype=torch.float64)
    sink = torch.zeros(2, dtype=torch.float64)
    want = R.talking_attention(q.expand(T, -1, -1), k, v, 1.0, 1e6, talk, sink, T, 0)[-1:]
    kc, vc = (torch.zeros(5, 2, 16, d, device=dev, dtype=dt) for _ in range(2))
    pos = torch.arange(T)
    kc[1 + pos // 16, :, pos % 16], vc[1 + pos // 16, :, pos % 16] = k.to(dev, dt), v.to(dev, dt)
    got = ops.talking_attention(q.to(dev, dt), kc, vc, batch_of([(T - 1, 1)], [[1, 2, 3, 4]], dev), talk.to(dev, dt), 1.0, 0.0, sink.float().to(dev), 0, 0)
    close(got, want, dt, limit=1e-3 if dt == torch.float32 else None)


@both
@pytest.mark.parametrize("H,G,d", [(16, 4, 128), (8, 2, 64), (32, 8, 128), (6, 2, 24)])
@pytest.mark.parametrize("shift", [-400.0, -130.0, 0.0, 130.0, 400.0])
def test_scores_of_any_size(dev, dt, H, G, d, shift):
    """Softmaxes of scores far from zero, of some rows and heads only: exponentials of the scores themselves would leave the range of fp32."""
    T, window, keep = 90, 40, 6
    q, k, v = rand(T, H, d, seed=1), rand(T, G, d, seed=2) * 0.1, rand(T, G, d, seed=3)
    q[..., 0], k[..., 0] = 0.0, 1.0
    q[::3, ::2, 0] = shift                                                   # every third query, every second head
    q, k = q.to(torch.bfloat16).double(), k.to(torch.bfloat16).double()
    talk, sink = torch.eye(H, dtype=torch.float64), rand(H, seed=4)
    talk[0, 1] = 0.5
    sink[2] = shift
    table = [4, 2, 7, 1, 3, 6]
    pos = torch.arange(T)
    at_page = torch.tensor(table)[pos // 16]
    kc, vc = (torch.zeros(8, G, 16, d, device=dev, dtype=dt) for _ in range(2))
    kc[at_page, :, pos % 16], vc[at_page, :, pos % 16] = k.to(dev, dt), v.to(dev, dt)
    for cap in (0.0, 1000.0):
        want = R.talking_attention(q, k, v, 1.0, cap or 1e9, talk, sink, window, keep)
        assert bool(want.isfinite().all())
        for portions, prefill in (([(0, T)], True), ([(50, 40)], True), ([(33, 1), (60, 1), (89, 1)], False)):
            rows = [p for a, n in portions for p in range(a, a + n)]
            got = ops.talking_attention(q[rows].contiguous().to(dev, dt), kc, vc, batch_of(portions, [table] * len(portions), dev, prefill, T), talk.to(dev, dt), 1.0, cap,
                                        sink.float().to(dev), window, keep)
            close(got, want[rows], dt, limit=1e-3 if dt == torch.float32 else 1.5e-2)


# ---------------------------------------------------------------------------------------------- whole models
def agrees(got, want, dt, slack=1.0, of=None):
    """``of`` (configuration, weights, tokens): in bf16, rows are left out where two experts' logits are so close that rounding chooses."""
    e = R.errors(got, want)
    if of is not None and dt == torch.bfloat16:
        keep = R.decided(*of)
        assert float(keep.float().mean()) > 0.6
        e = e * keep
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
        agrees(feed(eng, seq, tokens, sizes), want, dt, 3.0 if cfg is ODD and dt == torch.bfloat16 else 1.0, (cfg, w, tokens))   # narrow layers amplify rounding
        eng.release(seq)


class Watch:
    """Activation observer that keeps the stream behind every layer and may zero one."""

    def __new__(cls):
        from eredu_b200.runtime.inspection import ActivationObserver

        class Watching(ActivationObserver):
            def __init__(self):
                self.outputs, self.zero = {}, None

            def observe(self, name, value):
                self.outputs[name] = value.detach().double().cpu()

            def observe_moe_routing(self, observation):
                pass

            def intervene(self, name, value):
                return value * 0 if name == self.zero else None

        return Watching()


@both
def test_residual_stream_of_every_layer(dev, dt):
    w = R.weights(MIXED, seed=12)
    tokens = prompt(70, MIXED["vocab"], 5)
    want, layers = R.forward(MIXED, w, tokens, return_layers=True)
    eng = engine_for(MIXED, w, dev, dt)
    eng.model.observer = watch = Watch()
    agrees(feed(eng, eng.open_sequence(), tokens, [70]), want, dt, of=(MIXED, w, tokens))
    for i, x in enumerate(layers):
        close(watch.outputs[f"model.layers.{i}.output"], x, dt, limit=1e-4 if dt == torch.float32 else 3e-2)
    seq = eng.open_sequence()
    agrees(feed(eng, seq, tokens, [60, 1]), want, dt, of=(MIXED, w, tokens))                     # observed decode steps
    watch.zero = "model.layers.3.output"                                  # a stream somebody replaced is what the next layer reads
    assert R.error(feed(eng, eng.open_sequence(), tokens, [70]), want) > 0.1


@both
def test_first_tokens_and_one_token_prompts(dev, dt):
    w = R.weights(MIXED, seed=3)
    eng = engine_for(MIXED, w, dev, dt)
    for n in (1, 2, 3, 16, 17):
        tokens = prompt(n, MIXED["vocab"], n)
        seq = eng.open_sequence()
        agrees(feed(eng, seq, tokens, [n]), R.forward(MIXED, w, tokens), dt, of=(MIXED, w, tokens))
        eng.release(seq)


@both
def test_a_planted_mistake_would_show(dev, dt):
    """The same comparison with a mistake planted in the restatement is far outside the limit."""
    w = R.weights(MIXED, seed=1)
    tokens = prompt(90, MIXED["vocab"], 2)
    eng = engine_for(MIXED, w, dev, dt)
    got = feed(eng, eng.open_sequence(), tokens, [90])
    for layer, change in ((0, {"scale": 0.2}), (0, {"softcap": 4.0}), (2, {"mask": {"size": 25, "keep_first": 33}}), (4, {"mask": {"size": 33, "keep_first": 60}}),
                          (2, {"mask": {"size": 50, "keep_first": 0}})):
        other = json.loads(json.dumps(MIXED))
        other["layers"][layer]["mixer"].update(change)
        assert R.error(got, R.forward(other, w, tokens)) > 1.5 * LIMIT[dt], (layer, change)
    talk = w["l3.mix.talk"]
    for name, value in (("l0.canon1", w["l0.canon1"].flip(1)), ("l3.mix.talk", talk.t()), ("l3.mix.talk", torch.eye(12)), ("l2.mix.sink", w["l2.mix.sink"] - 9),
                        ("l0.ls1", w["l0.ls1"] * 0.5), ("l1.norm2", w["l1.norm2"] - 1), ("l0.mlp.act", w["l0.mlp.act"].flip(0)), ("l1.mlp.router.b", w["l1.mlp.router.b"] * -1),
                        ("l1.mlp.shared.down", w["l1.mlp.shared.down"] * 0), ("l4.mix.q.norm", w["l4.mix.q.norm"] * 0.3), ("final.norm", w["final.norm"] * 0)):
        assert R.error(got, R.forward(MIXED, dict(w, **{name: value}), tokens)) > 1.2 * LIMIT[dt], name


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
        agrees(torch.cat(got[i]), want[i], dt, of=(MIXED, w, reqs[i]))
    assert eng.kv.allocator.free_pages() == 19 and len(eng.kv._free_state_slots) == 3


@both
def test_long_decoding_across_windows_and_kept_tokens(dev, dt):
    w = R.weights(SMALL, seed=6)
    tokens = prompt(330, SMALL["vocab"], 7)
    eng = engine_for(SMALL, w, dev, dt, max_seq_len=336)
    agrees(feed(eng, eng.open_sequence(), tokens, [30, 1]), R.forward(SMALL, w, tokens), dt, of=(SMALL, w, tokens))


@both
def test_wide_layers(dev, dt):
    """Sizes that take the large tiles of every kernel: whole prompts of many rows, decode steps of several sequences."""
    cfg = R.config(512, 300, [R.attention_layer(16, 4, 128, 128, 70, 20, R.dense_ff(640), scale=0.08), R.attention_layer(32, 8, 64, 64, 33, 4, R.expert_ff(16, 4, 128, 256), scale=0.1)])
    w = R.weights(cfg, seed=2)
    reqs = [prompt(n, 300, n) for n in (300, 41, 130)]
    want = [R.forward(cfg, w, r, torch.float32) for r in reqs]
    eng = engine_for(cfg, w, dev, dt)
    seqs = [eng.open_sequence() for _ in reqs]
    heads = [290, 31, 120]
    first = eng.forward_tokens([(s, r[:n], range(n)) for s, r, n in zip(seqs, reqs, heads)]).split(heads)
    rest = [eng.forward_tokens([(s, [r[n + i]], [0]) for s, r, n in zip(seqs, reqs, heads)]) for i in range(10)]
    for i in range(3):
        agrees(torch.cat([first[i]] + [x[i:i + 1] for x in rest]), want[i], dt, of=(cfg, w, reqs[i]))


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
    assert report.is_loadable and report.model_type == "gulazen"
    prof = estimate_runtime_state(mc)
    assert prof.kv_bytes_per_token == 2 * sum(n * (a + b) for n, a, b in (mc.layer_kv_dims(i) for i in range(5)))
    assert prof.state_bytes_per_sequence == 4 * 5 * 3 * 96
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
    assert 0 < t["generated_tokens"] <= 6 and t["plan"]["model_type"] == "gulazen" and "TTFT" in capsys.readouterr().err


def test_random_models_of_a_configuration():
    from eredu_b200.models.llama import build_random, random_state

    mc = ModelConfig.from_hf_dict(SMALL)
    sd = random_state(mc, seed=3)
    a, b = build_from_tensors(mc, sd.__getitem__, sd.__contains__, "cpu", torch.float32), build_random(mc, "cpu", torch.float32, seed=3)
    assert torch.equal(a.layers[1].moe.w_down, b.layers[1].moe.w_down) and a.weight_bytes() > 0
    assert Engine(a, max_batch=1, max_seq_len=64).generate([[1, 2, 3]], SamplingParams(temperature=0.0), 4) == \
        Engine(b, max_batch=1, max_seq_len=64).generate([[1, 2, 3]], SamplingParams(temperature=0.0), 4)
