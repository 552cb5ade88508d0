"""Pulunex's sm_100a kernels: every mechanism alone and whole models through the engine, against the plain implementation."""
import types

import pytest
import torch

import pulunex_oracle as O
from pulunex_util import configs, feed, make_engine, portions, random_ids, row_error, sharp_model
from slopllm_b200.models.weights import ExpertWeights
from slopllm_b200.ops import experts as EX
from slopllm_b200.ops import get_ops
from slopllm_b200.ops import native as N
from slopllm_b200.ops import shift as SH
from slopllm_b200.ops import talking as TK
from test_zemezen_gpu import gen, rel, step_state

pytestmark = pytest.mark.gpu
CONFIGS = configs()
BF16_TOL, FP32_TOL = 0.06, 2e-5      # of the logits' spread
DTYPES = [torch.float32, torch.bfloat16]


def ops_of(dtype):
    return get_ops(types.SimpleNamespace(rms_norm_eps=1e-5), "cuda", None, dtype)


# ---- residual, norm and token shift ------------------------------------------------------------------------------------

@pytest.mark.parametrize("H", [1, 44, 256, 1001, 5120, 16384])
@pytest.mark.parametrize("dtype", DTYPES)
def test_token_shift(H, dtype):
    """Steps of portions and single tokens over reused, shuffled slots; long portions span several blocks of rows."""
    g = gen(H)
    total = [700, 41, 3, 1] if H < 2000 else [310, 41, 3, 1]
    y, r = ([torch.randn(n, H, generator=g) * s for n in total] for s in (3.0, 1.0))
    w, mix = torch.randn(1, generator=g).expand(H).contiguous(), torch.randn(H, generator=g)
    want = [O.token_shift(O.scalar_norm(a.double() + b.double(), w[0], 1e-3), mix) for a, b in zip(y, r)]
    state, slots = torch.full((6, H), 9.0, device="cuda"), [4, 0, 5, 2]
    done, got = [0] * 4, [[] for _ in total]
    for cut in ([total[0] - 15, 1, 2, 1], [1, 1, 1, 0], [2, 33, 0, 0], [9, 2, 0, 0], [1, 4, 0, 0], [2, 0, 0, 0]):
        live = [b for b in range(4) if cut[b]]
        rows = lambda x: torch.cat([x[b][done[b]:done[b] + cut[b]] for b in live]).cuda()
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")
        qo, bi = torch.tensor([0] + [cut[b] for b in live]).cumsum(0).to(torch.int32).cuda(), i32([j for j, b in enumerate(live) for _ in range(cut[b])])
        st = types.SimpleNamespace(positions=i32([done[b] + i for b in live for i in range(cut[b])]))
        out, res = SH.add_shift_norm(st, rows(y), rows(r), w.cuda(), 1e-3, SH.Shift(mix.cuda(), state, qo, i32([slots[b] for b in live]), bi), dtype)
        assert torch.equal(res, rows(y) + rows(r)) and out.dtype == dtype
        for j, b in enumerate(live):
            got[b].append(out[qo[j]:qo[j + 1]].cpu())
            done[b] += cut[b]
    assert done == total
    for b in range(4):
        assert rel(torch.cat(got[b]), want[b]) < (1e-6 if dtype == torch.float32 else 4e-3), b
    assert bool((state[[1, 3]] == 9).all())                        # slots of no sequence


@pytest.mark.parametrize("H", [1, 44, 1001, 2048])
@pytest.mark.parametrize("dtype", DTYPES)
def test_embedding_with_positions(H, dtype):
    g = gen(H)
    table, places, w, mix = torch.randn(9, H, generator=g).to(dtype), torch.randn(50, H, generator=g).to(dtype), torch.randn(H, generator=g), torch.randn(H, generator=g)
    ids, start, n = torch.tensor([3, 0, 8, 8, 1, 2, 4]), [0, 45], [2, 5]
    pos = torch.tensor([a + i for a, m in zip(start, n) for i in range(m)], dtype=torch.int32).cuda()
    st = types.SimpleNamespace(input_ids=ids.cuda(), positions=pos)
    r = table[ids].double() * 0.37 + places[pos.cpu().long()].double()
    h = O.rms(r, 1e-3) * w.double()
    before = torch.randn(H, generator=g)
    state = torch.stack([torch.ones(H), before]).cuda()
    shift = SH.Shift(mix.cuda(), state, torch.tensor([0, 2, 7], dtype=torch.int32).cuda(), torch.tensor([0, 1], dtype=torch.int32).cuda(),
                     torch.tensor([0, 0, 1, 1, 1, 1, 1], dtype=torch.int32).cuda())
    tol = 1e-6 if dtype == torch.float32 else 4e-3
    out, res = SH.embed_shift_norm(st, table.cuda(), 0.37, places.cuda(), w.cuda(), 1e-3, shift, dtype)
    assert rel(res, r) < 1e-6 and rel(out, torch.cat([O.token_shift(h[:2], mix), O.token_shift(h[2:], mix, before.double())])) < tol
    assert rel(state, h[[1, 6]]) < 1e-6
    for p in (places, None):
        out, res = SH.embed_shift_norm(st, table.cuda(), 0.37, None if p is None else p.cuda(), w.cuda(), 1e-3, None, dtype)
        x = r if p is not None else table[ids].double() * 0.37
        assert rel(res, x) < 1e-6 and rel(out, O.rms(x, 1e-3) * w.double()) < tol


# ---- feed-forwards ------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("I", [1, 13, 36, 1024, 3000])
@pytest.mark.parametrize("ti,to", [(torch.float32, torch.float32), (torch.float32, torch.bfloat16), (torch.bfloat16, torch.bfloat16)])
def test_activations(I, ti, to):
    g, ops, tol = gen(I), ops_of(to), 1e-6 if to == torch.float32 else 3e-3
    x, gate = (torch.randn(5, 2 * I, generator=g) * 3).to(ti), torch.randn(5, 4, generator=g) * 2
    out = torch.full((5, I + 3), 7.0, dtype=to, device="cuda")
    ops.plain_act(x.cuda()[:, :I], out[:, :I], "gelu_tanh")
    assert rel(out[:, :I], O.gelu_tanh(x[:, :I].double())) < tol and bool((out[:, I:] == 7).all())
    ops.gated_act(x.cuda(), out[:, :I], "silu", row_gate=gate.cuda()[:, 2])
    want = O.silu(x[:, :I].double()) * x[:, I:].double() * torch.sigmoid(gate[:, 2:3].double())
    assert rel(out[:, :I], want) < tol and bool((out[:, I:] == 7).all())


@pytest.mark.parametrize("E,top", [(1, 1), (7, 3), (32, 32), (33, 2), (140, 8), (1000, 20)])
def test_corrected_routing(E, top):
    g = gen(E)
    z, c = torch.randn(70, E + 5, generator=g) * 2, torch.randn(E, generator=g) * 0.7 - 0.4        # (choices below zero too)
    ids, w = EX.route_softmax(z.cuda()[:, 2:2 + E], top, correction=c.cuda())
    want, ww = O.choose(z[:, 2:2 + E].double(), c, top)
    assert torch.equal(ids.cpu().long(), want) and torch.allclose(w.cpu().double(), ww, atol=1e-6)
    plain, pw = EX.route_softmax(z.cuda()[:, 2:2 + E], top)
    want, ww = O.choose(z[:, 2:2 + E].double(), torch.zeros(E), top)
    assert torch.equal(plain.cpu().long(), want) and torch.allclose(pw.cpu().double(), ww, atol=1e-6)


def test_corrected_routing_in_groups():
    g = gen(3)
    z, c = torch.randn(50, 12, generator=g), torch.randn(12, generator=g) * 0.5 - 0.6
    ids, w = EX.route_softmax(z.cuda(), 4, 4, 2, c.cuda())
    a, b = EX.route_softmax(z, 4, 4, 2, c)
    assert torch.equal(ids.cpu(), a) and torch.allclose(w.cpu(), b, atol=1e-6)


@pytest.mark.parametrize("T", [1, 5, 32, 33, 150])
@pytest.mark.parametrize("E,extra,top,I,H", [(5, 3, 4, 13, 45), (8, 2, 3, 64, 128), (12, 20, 8, 24, 80), (3, 1, 2, 16, 48)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_experts_beside_identity_experts(T, E, extra, top, I, H, dtype):
    g = gen(T * E)
    x, out = torch.randn(T, H, generator=g).to(dtype), torch.randn(T, H, generator=g)
    w13, w2 = (torch.randn(E, 2 * I, H, generator=g) * H ** -0.5).to(dtype), (torch.randn(E, H, I, generator=g) * I ** -0.5).to(dtype)
    ids = torch.stack([torch.randperm(E + extra, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    ids[0] = torch.arange(E, E + top) if extra >= top else torch.arange(E + extra - top, E + extra)     # identity experts above all
    wts = torch.rand(T, top, generator=g)
    ex = ExpertWeights(w13.cuda(), w2.cuda())
    for identity in (True, False):
        want = out.double().clone()
        for t in range(T):
            for e, w in zip(ids[t].tolist(), wts[t].double()):
                xe = x[t].double()
                if e < E:
                    a, b = (w13[e].double() @ xe).chunk(2)
                    want[t] += w * (w2[e].double() @ (O.silu(a) * b))
                elif identity:
                    want[t] += w * xe
        got = out.cuda()
        EX.add_experts(x.cuda(), ex, ids.cuda(), wts.cuda(), got, ops_of(dtype), identity)
        assert rel(got - out.cuda(), want - out.double()) < (2e-5 if dtype == torch.float32 else 8e-3), identity


# ---- attention ----------------------------------------------------------------------------------------------------------

def attention_case(spans, heads, kv, dim, vdim, chunk, dtype, plant=None, seed=0, in_f32=False, ranks=1, scale=None, own_kv=True):
    """Portions `spans` = [(start, n)] over keys and values cached by earlier steps.  Both sides start from the same rows: the plain one
    rounds what is stored, so that differences are those of the scores, the softmax and the sums.  Returns (output, wanted)."""
    g, eps, r = gen(seed), 1e-4, heads // kv
    st, pt, slots = step_state(spans, seed)
    T, scale = len(st.positions), dim ** -0.5 if scale is None else scale
    sizes = (heads * dim, kv * dim, kv * vdim)
    proj = torch.randn(T, sum(sizes), generator=g).to(dtype)
    bias = torch.randn(sum(sizes), generator=g) * 0.5
    talk = (torch.eye(heads) + torch.randn(heads, heads, generator=g) * 0.7 * heads ** -0.5).to(torch.bfloat16).float()
    kc, vc = torch.zeros(slots, kv, dim, dtype=dtype), torch.zeros(slots, kv, vdim, dtype=dtype)
    old = [(O.rms(torch.randn(a, kv, dim, generator=g), eps).to(dtype), torch.randn(a, kv, vdim, generator=g).to(dtype)) for a, _ in spans]
    x, want, at = (proj.double() + bias.double()).split(sizes, 1), [], 0
    new_k, new_v = [], []
    for i, (a, n) in enumerate(spans):
        here, rows = torch.arange(a, a + n), slice(at, at + n)
        q = O.rms(x[0][rows].reshape(n, heads, dim), eps).to(dtype).double()
        k, v = O.rms(x[1][rows].reshape(n, kv, dim), eps).to(dtype), x[2][rows].reshape(n, kv, vdim).to(dtype)
        new_k.append(k), new_v.append(v)
        if plant is not None:
            plant(i, a, q, old[i][0], talk)
        for p in range(a + n):
            s = int(pt[i, p // 64]) * 64 + p % 64
            if p < a:
                kc[s], vc[s] = old[i][0][p], old[i][1][p]
            elif not own_kv:
                kc[s], vc[s] = k[p - a], v[p - a]
        keys, vals = torch.cat([old[i][0], k]).double().repeat_interleave(r, 1), torch.cat([old[i][1], v]).double().repeat_interleave(r, 1)
        w = O.softmax_over(O.talking_scores(q, keys, scale, talk), O.chunk_mask(here, torch.arange(a + n), chunk))
        want.append(torch.einsum("hts,shv->thv", w, vals).reshape(n, -1))
        at += n
    want, hl, kl = torch.cat(want), heads // ranks, kv // ranks
    out = torch.full((T, heads * vdim + 8), 5.0, dtype=dtype, device="cuda")
    for rk in range(ranks):
        shape = TK.TalkingShape(heads, kv, hl, kl, dim, vdim, scale, chunk, eps, own_kv)
        cut = lambda z: torch.cat([z[..., :sizes[0] + sizes[1]], z[..., sizes[0] + sizes[1] + rk * kl * vdim:sizes[0] + sizes[1] + (rk + 1) * kl * vdim]], -1)
        w = TK.TalkingWeights(cut(bias).cuda(), talk[rk * hl:(rk + 1) * hl].cuda(), torch.ones(dim, device="cuda"))
        kg, vg = kc.cuda(), vc[:, rk * kl:(rk + 1) * kl].contiguous().cuda()
        pg = cut(proj).cuda() if own_kv else proj[:, :sizes[0]].contiguous().cuda()
        q = TK.talking_pre(pg.float() if in_f32 else pg, shape, w, st, kg, vg, dtype)
        TK.talking_attention(q, shape, w, st, kg, vg, out[:, rk * hl * vdim:(rk + 1) * hl * vdim])
    assert bool((out[:, heads * vdim:] == 5).all())
    from slopllm_b200.ops import tcgen05
    tcgen05.check_errors(out.device)
    return out[:, :heads * vdim], want


def tol(dtype):
    return 2e-5 if dtype == torch.float32 else 6e-3


SHAPES = [(4, 2, 16, 16), (6, 2, 40, 24), (3, 3, 128, 128), (20, 1, 64, 136), (2, 1, 256, 200), (4, 2, 9, 14), (1, 1, 8, 2), (1, 1, 8, 8), (6, 3, 24, 48), (5, 5, 13, 10),
          (32, 8, 128, 128), (64, 8, 24, 16), (40, 4, 16, 136), (16, 16, 16, 32), (32, 32, 16, 16), (48, 3, 56, 24), (33, 11, 8, 8), (12, 12, 128, 64), (8, 4, 32, 256), (16, 16, 128, 128),
          (32, 16, 128, 120), (64, 8, 128, 128), (24, 12, 96, 88), (12, 4, 192, 192), (8, 8, 256, 248)]
SPANS = [[(0, 130), (70, 3), (200, 1), (5, 64)], [(150, 1), (3, 1), (0, 1), (256, 1)], [(127, 2)], [(0, 1)], [(300, 40)], [(0, 2), (64, 2), (63, 1)]]


@pytest.mark.parametrize("heads,kv,dim,vdim", SHAPES)
@pytest.mark.parametrize("chunk", [0, 64, 50, 1, 130])
@pytest.mark.parametrize("dtype", DTYPES)
def test_attention(heads, kv, dim, vdim, chunk, dtype):
    for i, spans in enumerate(SPANS):
        kw = [dict(), dict(in_f32=True), dict(own_kv=False, seed=3)][(i + chunk) % 3]
        got, want = attention_case(spans, heads, kv, dim, vdim, chunk, dtype, **kw)
        assert rel(got, want) < tol(dtype), (spans, kw)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim", [(6, 2, 24, 40), (32, 8, 64, 64), (8, 2, 16, 24)])
def test_attention_of_shared_heads(heads, kv, dim, vdim, dtype):
    """Two emulated ranks: all query and key heads, half of the output and value heads each."""
    for spans in SPANS[:2]:
        got, want = attention_case(spans, heads, kv, dim, vdim, 60, dtype, ranks=2)
        assert rel(got, want) < tol(dtype), spans


def test_sizes_on_the_tensor_cores():
    """The sizes above take the kernel that they are meant for."""
    on = [s for s in SHAPES if N.fn("sl_talking_queries")(s[0], s[1], s[0], s[1], s[2], s[3], 0)]
    assert (32, 8, 128, 128) in on and (64, 8, 24, 16) in on and (3, 3, 128, 128) in on and (2, 1, 256, 200) in on and (1, 1, 8, 8) in on
    assert (32, 32, 16, 16) not in on and (4, 2, 9, 14) not in on
    assert all(N.fn("sl_talking_queries")(s[0], s[1], s[0], s[1], s[2], s[3], 1) == 1 for s in on)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim", [(4, 2, 16, 24), (1, 1, 16, 14), (32, 8, 64, 32)])
def test_one_far_key(heads, kv, dim, vdim, dtype):
    """One cached key answers the query far better than all others: at the chunk's first position it decides, right in front of it it is
    not seen; also around page borders, hundreds of tokens back and directly in front."""
    def planted(key, factor=1.0):
        def plant(b, start, q, keys, talk):
            for h in range(kv):                                    # every head's mixture leans to it
                mean = q[0, h * (heads // kv):(h + 1) * (heads // kv)].sum(0)
                keys[min(key, start - 1), h] = (mean / mean.norm() * dim ** 0.5 * 6 * factor).to(keys.dtype)
        return plant

    for chunk in (0, 64, 512, 300):
        for key in (0, 1, 63, 64, 127, 128, 299, 300, 301, 447, 448, 511):
            for spans in ([(511, 1), (512, 1), (577, 1)], [(512, 2)], [(513, 70), (511, 1)]):
                got, want = attention_case(spans, heads, kv, dim, vdim, chunk, dtype, plant=planted(key), seed=key, scale=0.5)
                assert rel(got, want) < 2 * tol(dtype), (chunk, key, spans)
    # the plant shows exactly inside the chunk
    for key, chunk, seen in ((448, 64, True), (447, 64, False), (300, 300, True), (299, 300, False), (0, 0, True), (0, 512, True), (0, 511, False)):
        a, _ = attention_case([(511, 1)], heads, kv, dim, vdim, chunk, dtype, plant=planted(key), seed=1, scale=0.5)
        b, _ = attention_case([(511, 1)], heads, kv, dim, vdim, chunk, dtype, plant=planted(key, -1.0), seed=1, scale=0.5)
        assert (rel(a, b) > 0.1) == seen and (seen or torch.equal(a, b)), (key, chunk)


@pytest.mark.parametrize("dim", range(8, 137, 8))
def test_every_size_of_whole_pieces(dim):
    for i, vdim in enumerate((8, 24, 40, 56, 64, 88, 104, 136)):
        kv = 1 + i % 3
        for spans in ([(70, 1), (5, 1), (128, 1)], [(20, 70), (66, 2)]):
            got, want = attention_case(spans, (1 + i % 4) * kv, kv, dim, vdim, 100 if i % 2 else 0, torch.bfloat16, seed=vdim)
            assert rel(got, want) < tol(torch.bfloat16), (vdim, spans)


def test_key_splits():
    """Long contexts: the keys of one query tile are shared by several blocks."""
    for heads, kv, dim, vdim in ((8, 2, 64, 64), (32, 8, 128, 128), (40, 4, 16, 136)):
        for spans in ([(1500, 1), (700, 1)], [(1999, 1)], [(64 * i + 5, 1) for i in range(40)], [(1900, 20), (600, 1)], [(1990, 2)]):
            for chunk in (0, 700, 1024):
                got, want = attention_case(spans, heads, kv, dim, vdim, chunk, torch.bfloat16)
                assert rel(got, want) < tol(torch.bfloat16), (heads, spans, chunk)
    assert TK.key_splits(1, 2048, 32) == 64 and TK.key_splits(600, 4096, 32) == 1 and TK.key_splits(1, 1, 32) == 1


def test_results_do_not_depend_on_the_cut():
    """The same query in a long portion, in a short one and decoded."""
    a, _ = attention_case([(190, 10)], 32, 8, 64, 64, 128, torch.bfloat16, own_kv=False, seed=2)
    b, want = attention_case([(190, 10)], 32, 8, 64, 64, 128, torch.float32, own_kv=False, seed=2)
    assert rel(b, want) < 2e-5 and rel(a, b) < 3e-2


# ---- whole models through the engine ----------------------------------------------------------------------------------

def within(err, dtype):
    """(a routed token whose choice is close may go to another expert in bf16: single rows get more room than the rest)"""
    if dtype == torch.float32:
        return bool(err.max() < FP32_TOL)
    return bool(err.median() < BF16_TOL / 2 and (err > 2 * BF16_TOL).double().mean() < 0.1)


@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", DTYPES)
def test_engine_schedules(name, dtype):
    """Whole prompt, portions down to two tokens, token by token: all positions against the plain forward."""
    raw = CONFIGS[name]
    t = O.random_tensors(raw, 1)
    ids = random_ids(raw, 200, 2)
    want = O.forward(raw, t, ids)
    eng = make_engine(raw, t, "cuda", dtype)
    for cuts in ([200], portions(200, [2, 64, 3, 29, 70]), portions(200, [150], tail=40), [2] * 100, [1] * 200):
        err = row_error(feed(eng, ids, cuts), want)
        assert within(err, dtype), (cuts[:5], err.argmax(), err.max(), err.median())


@pytest.mark.parametrize("dtype", DTYPES)
def test_engine_mixed_batches_and_reused_slots(dtype):
    raw = CONFIGS["tiled"]
    t = O.random_tensors(raw, 3)
    eng = make_engine(raw, t, "cuda", dtype, num_pages=10, max_states=3, max_batch=3)
    lens = [170, 40, 129, 7, 64, 190, 3, 90]
    ids = [random_ids(raw, n, 10 + i) for i, n in enumerate(lens)]
    got = [[] for _ in lens]
    live, waiting, turn = {}, list(range(len(lens))), 0
    while live or waiting:
        while waiting and len(live) < 3:
            live[waiting.pop(0)] = eng.kv.new_sequence()
        step = [(i, s, ids[i][s.length:s.length + [17, 1, 2, 66, 1, 64, 1, 1, 1, 3][(turn + j * 3) % 10]]) for j, (i, s) in enumerate(live.items())]
        out = eng.step([s for _, s, _ in step], [x for _, _, x in step], [range(len(x)) for _, _, x in step]).cpu()
        at = 0
        for i, s, x in step:
            got[i].append(out[at:at + len(x)])
            at += len(x)
            if s.length == lens[i]:
                eng.finish(live.pop(i))
        turn += 1
    eng.kv.assert_clear()
    for i in range(len(lens)):
        assert within(row_error(torch.cat(got[i]), O.forward(raw, t, ids[i])), dtype), i
        alone = feed(eng, ids[i], [lens[i]])                      # the same request alone
        assert within(row_error(torch.cat(got[i]), alone), dtype), i


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    """Hundreds of decoded tokens over page and chunk borders, in a graph."""
    raw, t = sharp_model()
    ids = random_ids(raw, 420, 6)
    want = O.forward(raw, t, ids)
    changed = O.forward(raw, t, [(ids[0] + 1) % raw["vocab"]] + ids[1:])
    assert row_error(changed, want)[-1] > 1e-3                    # the first token still matters at the end
    err = row_error(feed(make_engine(raw, t, "cuda", dtype), ids, [60] + [1] * 360), want)
    assert within(err, dtype), (err.argmax(), err.max(), err.median())


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_scheduler(dtype):
    from slopllm_b200.config import SamplingParams
    from slopllm_b200.sampling.workspace import SamplingWorkspace
    from slopllm_b200.scheduler.scheduler import GenerationRequest, GenerationScheduler
    raw = CONFIGS["tiled"]
    t = O.random_tensors(raw, 7)
    eng = make_engine(raw, t, "cuda", dtype, num_pages=14, max_batch=3, max_states=3)
    eng.sampler = SamplingWorkspace(eng.device, raw["vocab"], seed=0)
    sched = GenerationScheduler(eng, max_batch=3, chunk_size=48)
    reqs = [GenerationRequest(id=str(i), input_ids=random_ids(raw, n, 20 + i), max_tokens=8, sampling=SamplingParams(temperature=0.0))
            for i, n in enumerate((150, 3, 25, 100, 1, 30, 64))]
    for r in reqs:
        sched.submit(r)
    for _ in range(300):
        sched.step()
        if all(r.retired for r in reqs):
            break
    for r in reqs:
        assert r.error is None and len(r.generated) == 8
        logits = O.forward(raw, t, r.input_ids + r.generated)[len(r.input_ids) - 1:-1]
        best = logits.max(-1).values
        took = logits.gather(-1, torch.tensor(r.generated)[:, None]).squeeze(-1)
        assert (best - took).max() <= (1e-4 if dtype == torch.float32 else 0.4) * logits.std(), r.id
    assert eng.model.states.free == 3
