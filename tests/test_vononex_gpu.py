"""Vononex's sm_100a kernels: every mechanism alone and whole models through the engine, against the plain implementation."""
import types

import pytest
import torch

import vononex_oracle as O
from slopllm_b200.ops import get_ops
from slopllm_b200.ops import grouped as G
from slopllm_b200.ops import recurrent as RC
from slopllm_b200.ops.rotary import AngleTable, adjacent_order
from test_zemezen_gpu import gen, rel, step_state
from vononex_util import configs, far_key_model, feed, make_engine, portions, random_ids, row_error

pytestmark = pytest.mark.gpu
CONFIGS = configs()
BF16_TOL, FP32_TOL = 0.06, 1e-5      # of the logits' spread
DTYPES = [torch.float32, torch.bfloat16]


def ops_of(dtype):
    return get_ops(types.SimpleNamespace(rms_norm_eps=1e-5), "cuda", None, dtype)


# ---- residual, norms, activation, angles ------------------------------------------------------------------------------

@pytest.mark.parametrize("H", [1, 44, 256, 1001, 5120, 16384])
@pytest.mark.parametrize("dtype", DTYPES)
def test_norm_of_the_sum(H, dtype):
    g, ops = gen(H), ops_of(dtype)
    y, r, w, nxt, b = torch.randn(7, H, generator=g) * 3, torch.randn(7, H, generator=g), *(torch.randn(H, generator=g) for _ in range(3))
    for bias in (None, b):
        for last in (None, nxt):
            out, res = ops.sum_norm(y.cuda(), r.cuda(), 1.7, None if bias is None else bias.cuda(), w.cuda(), None if last is None else last.cuda(), 1e-3)
            want = O.norm(1.7 * r.double() + y.double() + (0 if bias is None else bias.double()), w, 1e-3)
            assert rel(res, want) < 1e-6 and out.dtype == dtype and res.dtype == torch.float32
            assert rel(out, want if last is None else O.norm(want, last, 1e-3)) < (1e-6 if dtype == torch.float32 else 4e-3)
    table = torch.randn(9, H, generator=g).to(dtype)
    ids = torch.tensor([3, 0, 8, 8])
    out, res = ops.embed_rows(ids.cuda(), table.cuda())
    assert torch.equal(res.cpu(), table[ids].float()) and torch.equal(out.cpu(), table[ids])


@pytest.mark.parametrize("I", [1, 13, 36, 1024, 3000])
@pytest.mark.parametrize("ti,to", [(torch.float32, torch.float32), (torch.float32, torch.bfloat16), (torch.bfloat16, torch.bfloat16)])
def test_gelu_activation_with_biases(I, ti, to):
    x = (torch.randn(5, 2 * I, generator=gen(I)) * 3).to(ti)
    b = torch.randn(2 * I, generator=gen(1))
    out = torch.empty(5, I, dtype=to, device="cuda")
    for bias in (None, b):
        ops_of(to).gated_act(x.cuda(), out, "gelu_tanh", None if bias is None else bias.cuda())
        z = x.double() + (0 if bias is None else bias.double())
        assert rel(out, O.gelu_tanh(z[:, :I]) * z[:, I:]) < (1e-6 if to == torch.float32 else 3e-3)


def test_angles_keep_their_accuracy_far_out():
    table = AngleTable()
    turns = [table.turn(2, 10.0), table.turn(128, 1e4), table.turn(48, 1e6)]
    pos = torch.tensor([0, 1, 63, 64, 1000, 131071, 10 ** 6], dtype=torch.int32)
    got = table.at(pos.cuda()).cpu().double()
    for t, base in zip(turns, (10.0, 1e4, 1e6)):
        a = pos.double()[:, None] * base ** (-2.0 * torch.arange(t.dims // 2, dtype=torch.float64) / t.dims)
        assert (t.columns(got)[..., 0] - a.cos()).abs().max() < 5e-7 and (t.columns(got)[..., 1] - a.sin()).abs().max() < 5e-7


# ---- attention with whole-row norms and turned values -----------------------------------------------------------------

def attention_case(spans, heads, kv, dim, vdim, dims, dtype, plant=None, seed=0, in_f32=False, out_scale=1.0, ranks=1, bias=True):
    """Portions `spans` = [(start, n)] over keys and values cached by earlier steps.  `ranks`: the heads are shared by that many
    emulated ranks, whose sums of squares are added.  Returns (output, wanted)."""
    g, eps, base = gen(seed), 1e-4, 3e3
    st, pt, slots = step_state(spans, seed)
    T, scale = len(st.positions), dim ** -0.5
    sizes = (heads * dim, kv * dim, kv * vdim)
    proj = torch.randn(T, sum(sizes), generator=g).to(dtype)
    b = torch.randn(sum(sizes), generator=g) * (0.5 if bias else 0.0)
    qn, kn = torch.randn(sizes[0], generator=g) * 0.2 + 1, torch.randn(sizes[1], generator=g) * 0.2 + 1
    temp = torch.randn(heads, generator=g) * 0.3 + 1
    kc, vc = torch.zeros(slots, kv, dim, dtype=dtype), torch.zeros(slots, kv, vdim, dtype=dtype)
    old = [(torch.randn(a, kv, dim, generator=g).to(dtype), torch.randn(a, kv, vdim, generator=g).to(dtype)) for a, _ in spans]
    x, want, at = (proj.double() + b.double()).split(sizes, 1), [], 0
    for i, (a, n) in enumerate(spans):
        here, rows = torch.arange(a, a + n), slice(at, at + n)
        q = O.rotate(O.norm(x[0][rows], qn, eps).view(n, heads, dim), here, dims, base)
        k = O.rotate(O.norm(x[1][rows], kn, eps).view(n, kv, dim), here, dims, base)
        if plant is not None:
            plant(i, a, q * temp.double()[:, None], old[i][0])
        for p in range(a):
            s = int(pt[i, p // 64]) * 64 + p % 64
            # the caches hold every head in adjacent order; cached values are turned already
            kc[s], vc[s] = old[i][0][p][:, adjacent_order(dim, dims)], old[i][1][p][:, adjacent_order(vdim, vdim)]
        keys = torch.cat([old[i][0].double(), k]).repeat_interleave(heads // kv, 1)
        v = torch.cat([old[i][1].double(), O.rotate(x[2][rows].reshape(n, kv, vdim), here, vdim, base)]).repeat_interleave(heads // kv, 1)
        w = O.causal_softmax(torch.einsum("thd,shd->hts", q, keys) * scale * temp.double()[:, None, None])
        want.append(O.rotate(torch.einsum("hts,shv->thv", w, v), here, vdim, base, -1.0).reshape(n, -1) * out_scale)
        at += n

    table = AngleTable()
    table.turn(14, 77.0)                                          # other rotations in front of these
    turn, v_turn = table.turn(dims, base), table.turn(vdim, base)
    angles = table.of(st)
    order = lambda t, h, d, k: t.view(*t.shape[:-1], h, d)[..., adjacent_order(d, k)].flatten(-2)
    stored = lambda t: [order(y, h, d, k) for y, h, d, k in zip(t.split(sizes, -1), (heads, kv, kv), (dim, dim, vdim), (dims, dims, vdim))]
    parts, biases = stored(proj), stored(b)
    out = torch.full((T, heads * vdim + 8), 5.0, dtype=dtype, device="cuda")
    hl, kl = heads // ranks, kv // ranks
    shape = G.GroupedShape(hl, kl, dim, vdim, scale, eps=eps)
    cut = lambda t, h, d, r: t[..., r * h * d // ranks:(r + 1) * h * d // ranks]
    x0 = stored(proj.double() + b.double())                       # (sums of all ranks, as the reduction would give them)
    sums = torch.stack([x0[0].square().sum(-1), x0[1].square().sum(-1)], -1).float()
    own = []

    class Comm:
        ctx = types.SimpleNamespace(world=ranks)

        def all_reduce(self, s):
            own.append(s.cpu())
            return sums.cuda()

    for r in range(ranks):
        pick = lambda ts: torch.cat([cut(t, h, d, r) for t, h, d in zip(ts, (heads, kv, kv), (dim, dim, vdim))], -1)
        w = G.RowNormWeights(cut(order(qn, heads, dim, dims), heads, dim, r).cuda(), cut(order(kn, kv, dim, dims), kv, dim, r).cuda(),
                             pick(biases).cuda() if bias else None, temp[r * hl:(r + 1) * hl].cuda())
        kg, vg = kc[:, r * kl:(r + 1) * kl].contiguous().cuda(), vc[:, r * kl:(r + 1) * kl].contiguous().cuda()
        pg = pick(parts).cuda()
        q = G.grouped_row_pre(pg.float() if in_f32 else pg, shape, w, turn, v_turn, angles, st, kg, vg, dtype, Comm() if ranks > 1 else None)
        view = out[:, r * hl * vdim:(r + 1) * hl * vdim]
        G.grouped_attention(q, shape, w, st, kg, vg, view, G.Finish(v_turn, angles, out_scale))
    if ranks > 1:
        assert rel(sum(own), sums) < 1e-5
    assert bool((out[:, heads * vdim:] == 5).all())
    back = torch.argsort(adjacent_order(vdim, vdim))
    return out[:, :heads * vdim].reshape(T, heads, vdim)[..., back.cuda()].reshape(T, -1), torch.cat(want)


SHAPES = [(4, 2, 16, 16, 8), (6, 2, 40, 24, 40), (3, 3, 128, 128, 128), (20, 1, 64, 136, 64), (2, 1, 256, 200, 2), (4, 2, 9, 14, 6), (1, 1, 8, 2, 2),
          (6, 3, 24, 48, 24), (5, 5, 13, 10, 12)]
SPANS = [[(0, 130), (70, 3), (200, 1), (5, 64)], [(150, 1), (3, 1), (0, 1), (256, 1)], [(127, 2)], [(0, 1)], [(300, 40)], [(0, 2), (64, 2), (63, 1)]]


@pytest.mark.parametrize("heads,kv,dim,vdim,dims", SHAPES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_attention(heads, kv, dim, vdim, dims, dtype):
    for spans in SPANS:
        for kw in (dict(), dict(in_f32=True, out_scale=-1.3), dict(bias=False, seed=3)):
            got, want = attention_case(spans, heads, kv, dim, vdim, dims, dtype, **kw)
            assert rel(got, want) < (2e-5 if dtype == torch.float32 else 1.2e-2), (spans, kw)


@pytest.mark.parametrize("dtype", DTYPES)
def test_attention_of_shared_heads(dtype):
    for spans in SPANS[:2]:
        got, want = attention_case(spans, 6, 2, 24, 40, 16, dtype, ranks=2)
        assert rel(got, want) < (2e-5 if dtype == torch.float32 else 1.2e-2), spans


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("vdim", [16, 24, 14])
def test_one_far_key(vdim, dtype):
    """One cached key answers the query far better than all others: at the sequence's start, around page borders, hundreds of tokens back
    and directly in front.  Its value must come back turned by its own distance."""
    for key in (0, 1, 63, 64, 127, 128, 400, 511):
        def plant(b, start, q, keys):
            keys[min(key, start - 1)] = (q[0].mean(0, keepdim=True) * 14.0).to(keys.dtype).expand_as(keys[0])

        for spans in ([(512, 1), (577, 1), (640, 1)], [(512, 2)], [(513, 70), (520, 1)]):
            got, want = attention_case(spans, 1, 1, 16, vdim, 16, dtype, plant=plant, seed=key)
            assert rel(got, want) < (2e-5 if dtype == torch.float32 else 1.5e-2), (key, spans)
    a, _ = attention_case([(512, 1)], 1, 1, 16, vdim, 16, dtype, plant=plant, seed=key)
    b, _ = attention_case([(512, 1)], 1, 1, 16, vdim, 16, dtype, seed=key)
    assert rel(a, b) > 0.2                                        # the planted key decides the row


@pytest.mark.parametrize("dim", range(8, 137, 8))
def test_every_size_of_whole_pieces(dim):
    """Heads of every multiple of eight values, decoded and in portions: rows of a tile are copied by lanes that share them unevenly."""
    for i, vdim in enumerate((8, 24, 40, 56, 64, 88, 104, 136)):
        kv = 1 + i % 2
        for spans in ([(70, 1), (5, 1), (128, 1)], [(20, 70), (66, 2)]):
            got, want = attention_case(spans, 2 * kv, kv, dim, vdim, dim - 8 * (i % 2) if dim > 8 else dim, torch.bfloat16, seed=vdim)
            assert rel(got, want) < 1.2e-2, (vdim, spans)


def test_decode_key_splits():
    """Long contexts: the keys of one row are shared by several blocks, whose sum is turned back once."""
    for spans in ([(1500, 1), (700, 1)], [(1999, 1)], [(64 * i + 5, 1) for i in range(40)]):
        got, want = attention_case(spans, 8, 2, 64, 64, 64, torch.bfloat16, out_scale=0.5)
        assert rel(got, want) < 1.2e-2


# ---- retention ----------------------------------------------------------------------------------------------------------

def retention_case(lens, h, dk, dv, dims, dtype, decay, seed=0, fresh=False, in_f32=False):
    """Portions behind earlier tokens, from a non-zero state; returns (arguments, wanted output, wanted states)."""
    g, B, T = gen(seed), len(lens), sum(lens)
    start = [0 if fresh else 5 + 37 * b for b in range(B)]
    pos = torch.cat([torch.arange(a, a + n) for a, n in zip(start, lens)])
    proj = torch.randn(T, h * (2 * dk + 2 * dv), generator=g).to(dtype)
    slots = [(2 * b + 1) % (B + 2) for b in range(B)] if (B + 2) % 2 else list(range(B))[::-1]
    S = torch.zeros(B + 2, h, dk, dv)
    order, want, S_want, at = adjacent_order(dk, dims), [], {}, 0
    q, k, v, gate = proj.double().split([h * dk, h * dk, h * dv, h * dv], 1)
    for b, n in enumerate(lens):
        r = slice(at, at + n)
        if not fresh:
            S[slots[b]] = torch.randn(h, dk, dv, generator=g)
        turned = lambda y: O.rotate(y[r].reshape(n, h, dk), pos[r], dims, 200.0)
        back = S[slots[b]][:, torch.argsort(order)].double()      # (states hold keys in adjacent order, and unscaled)
        o, s = O.retain(turned(q) * dk ** -0.5, turned(k), v[r].reshape(n, h, dv), torch.tensor(decay, dtype=torch.float64), back)
        S_want[slots[b]] = s[:, order]
        want.append(O.rms(o, 1e-3).reshape(n, -1) * O.silu(gate[r]) * 1.25)
        at += n
    for i in range(2 * h):
        proj[:, i * dk:(i + 1) * dk] = proj[:, i * dk:(i + 1) * dk][:, order]
    table = AngleTable()
    table.turn(6, 77.0)
    turn = table.turn(dims, 200.0)
    ind = torch.tensor([0] + lens).cumsum(0).to(torch.int32)
    args = ((proj.float() if in_f32 else proj).cuda(), RC.retention_decays(decay).cuda(), turn, table.at(pos.to(torch.int32).cuda()), S.cuda(), ind.cuda(),
            torch.tensor(slots, dtype=torch.int32).cuda(), (h, dk, dv))
    return args, torch.cat(want), S_want


def run_retention(args, dtype, plan):
    proj, decay, turn, angles, S, ind, slots, (h, dk, dv) = args
    S, wide = S.clone(), torch.full((proj.shape[0], h * dv + 8), 5.0, dtype=dtype, device="cuda")
    RC.retention_mix(proj, decay, turn, angles, 1e-3, S, ind, slots, h, dk, dv, wide[:, :h * dv], 1.25, plan)
    assert bool((wide[:, h * dv:] == 5).all())
    return wide[:, :h * dv], S


RETENTIONS = [([200, 1, 64, 17], 2, 32, 48, 32), ([130], 3, 128, 128, 128), ([65, 63, 3], 4, 40, 24, 16), ([33, 2], 2, 10, 7, 6), ([70], 2, 24, 160, 8),
              ([1, 1, 1], 4, 64, 32, 64), ([1, 1], 2, 9, 13, 8), ([1], 2, 128, 128, 64), ([129], 2, 136, 96, 128), ([1], 1, 200, 264, 2), ([192, 128], 2, 16, 8, 16),
              ([16, 2, 1], 1, 8, 8, 2), ([64], 2, 256, 256, 256)]


@pytest.mark.parametrize("lens,h,dk,dv,dims", RETENTIONS)
@pytest.mark.parametrize("decays", [[0.9, 0.99, 0.5, 0.999], [1.0, 0.0, 0.9995, 0.1]])
@pytest.mark.parametrize("dtype", DTYPES)
def test_retention(lens, h, dk, dv, dims, decays, dtype):
    for in_f32 in ((False, True) if dtype == torch.bfloat16 else (False,)):
        args, want, S_want = retention_case(lens, h, dk, dv, dims, dtype, decays[:h], seed=dk, in_f32=in_f32)
        plans = [None] + ([RC.ChunkPlan(lens, "cuda")] if dtype == torch.bfloat16 and max(lens) >= RC.CHUNK_MIN_Q and not in_f32 else [])
        for plan in plans:
            got, S = run_retention(args, dtype, plan)
            for slot, x in S_want.items():
                assert rel(S[slot], x) < 1e-5, plan
            assert rel(got, want) < (2e-5 if dtype == torch.float32 else 4e-3), plan


@pytest.mark.parametrize("dk", range(8, 137, 8))
def test_retention_of_every_size_of_whole_pieces(dk):
    for i, dv in enumerate((8, 24, 40, 56, 64, 88, 136)):
        args, want, S_want = retention_case([70, 1, 18], 2, dk, dv, dk - 2 * (i % 3), torch.bfloat16, [0.97, 0.999], seed=dv)
        for plan in (None, RC.ChunkPlan([70, 1, 18], "cuda")):
            got, S = run_retention(args, torch.bfloat16, plan)
            assert all(rel(S[slot], x) < 1e-5 for slot, x in S_want.items()) and rel(got, want) < 4e-3, (dv, plan)


def test_retention_chunks_follow_the_step_kernel():
    """Long portions of slow decays, also in several passes over the chunks: 32-bit sums on the tensor cores."""
    args, _, _ = retention_case([500, 90, 64], 2, 64, 80, 64, torch.bfloat16, [0.9998, 1.0], seed=5, fresh=True)
    a, S = run_retention(args, torch.bfloat16, None)
    for budget in (96 << 20, 3 * 2 * 64 * 80 * 4):
        old, RC.CHUNK_SCRATCH_BYTES = RC.CHUNK_SCRATCH_BYTES, budget
        try:
            b, Sc = run_retention(args, torch.bfloat16, RC.ChunkPlan([500, 90, 64], "cuda"))
        finally:
            RC.CHUNK_SCRATCH_BYTES = old
        assert rel(Sc, S) < 1e-5 and rel(b, a) < 3e-3


# ---- minGRU -------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("W", [1, 37, 64, 520, 2048])
@pytest.mark.parametrize("dtype", DTYPES)
def test_min_gru(W, dtype):
    """Sequences in portions of every size, their states in reused, shuffled slots."""
    g = gen(W)
    total = [210, 41, 7, 1]
    x = [(torch.randn(n, 3 * W, generator=g) * 2).to(dtype) for n in total]
    bias = torch.randn(2 * W, generator=g)
    want = []
    for y in x:
        z, u, gate = y.double().split(W, 1)
        want.append(O.min_gru(torch.sigmoid(z + bias[:W]), u + bias[W:], torch.zeros(W, dtype=torch.float64)) * O.silu(gate))
    state, slots = torch.zeros(6, W, device="cuda"), [4, 0, 5, 2]
    done, got = [0] * 4, [[] for _ in total]
    for cut in ([66, 1, 2, 1], [1, 1, 1, 0], [2, 33, 3, 0], [127, 2, 1, 0], [1, 4, 0, 0], [13, 0, 0, 0]):
        live = [b for b in range(4) if cut[b]]
        lens = [cut[b] for b in live]
        rows = torch.cat([x[b][done[b]:done[b] + cut[b]] for b in live])
        ind = torch.tensor([0] + lens).cumsum(0).to(torch.int32)
        plan = RC.ChunkPlan(lens, "cuda") if max(lens) > 1 else None
        y = RC.min_gru_mix((rows.float() if len(live) == 3 else rows).cuda(), bias.cuda(), state, ind.cuda(),
                           torch.tensor([slots[b] for b in live], dtype=torch.int32).cuda(), W, dtype, plan).cpu()
        for j, b in enumerate(live):
            got[b].append(y[ind[j]:ind[j + 1]])
            done[b] += cut[b]
    assert done == total
    for b in range(4):
        assert rel(torch.cat(got[b]), want[b]) < (2e-6 if dtype == torch.float32 else 3e-3), b
    assert not state[1].any() and not state[3].any()


def test_min_gru_without_biases_and_with_long_memory():
    W, n = 96, 1500
    g = gen(0)
    x = torch.randn(n, 3 * W, generator=g)
    x[:, :W] -= 7                                                 # a token changes a thousandth of the state
    z, u, gate = x.double().split(W, 1)
    want = O.min_gru(torch.sigmoid(z), u, torch.zeros(W, dtype=torch.float64)) * O.silu(gate)
    state, one = torch.zeros(1, W, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
    y = RC.min_gru_mix(x.cuda(), None, state, torch.tensor([0, n], dtype=torch.int32).cuda(), one, W, torch.float32, RC.ChunkPlan([n], "cuda"))
    assert rel(y, want) < 2e-6


# ---- whole models through the engine ----------------------------------------------------------------------------------

def within(err, dtype):
    """(single rows whose retention heads nearly cancel show rounding enlarged)"""
    tol = FP32_TOL if dtype == torch.float32 else BF16_TOL / 2
    return bool(err.mean() < tol and (err > 4 * tol).double().mean() < 0.03 and err.max() < 60 * tol)


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
        assert within(err, dtype), (cuts[:5], err.argmax(), err.max(), err.mean())


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
        err = row_error(torch.cat(got[i]), O.forward(raw, t, ids[i]))
        tol = FP32_TOL if dtype == torch.float32 else BF16_TOL / 2
        assert err.median() < tol and (err > 4 * tol).double().mean() < 0.2, (i, err.max(), err.mean())
        alone = torch.cat([feed(eng, ids[i], [lens[i]])])         # the same request alone
        assert row_error(torch.cat(got[i]), alone).median() < tol


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixers_of_a_layer_in_turn_give_the_same(dtype, monkeypatch):
    """A second stream for one of the two mixers changes no result."""
    from slopllm_b200.models import mixers
    raw = CONFIGS["tiled"]
    t = O.random_tensors(raw, 5)
    ids = random_ids(raw, 150, 8)
    cuts = portions(150, [70, 3], tail=30)
    a = feed(make_engine(raw, t, "cuda", dtype), ids, cuts)
    monkeypatch.setattr(mixers, "TOGETHER_MAX", 0)
    assert torch.equal(a, feed(make_engine(raw, t, "cuda", dtype), ids, cuts))


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    """Hundreds of decoded tokens over page borders, in a graph."""
    raw, t = far_key_model()
    ids = random_ids(raw, 420, 6)
    want = O.forward(raw, t, ids)
    changed = O.forward(raw, t, [(ids[0] + 1) % raw["vocab"]] + ids[1:])
    assert row_error(changed, want)[-1] > 2e-3                    # the first token still matters at the end
    err = row_error(feed(make_engine(raw, t, "cuda", dtype), ids, [60] + [1] * 360), want)
    assert within(err, dtype), (err.argmax(), err.max(), err.mean())


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_scheduler(dtype):
    from slopllm_b200.config import SamplingParams
    from slopllm_b200.sampling.workspace import SamplingWorkspace
    from slopllm_b200.scheduler.scheduler import GenerationRequest, GenerationScheduler
    raw = CONFIGS["wide"]
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
        assert (best - took).max() <= (1e-4 if dtype == torch.float32 else 0.3) * logits.std(), r.id
    assert eng.model.states.free == 3
