"""Zemezen's sm_100a kernels: every mechanism alone and whole models through the engine, against the plain implementation."""
import types

import pytest
import torch

import zemezen_oracle as O
from slopllm_b200.models.glm_moe_dsa import StepState
from slopllm_b200.models.weights import ExpertWeights
from slopllm_b200.ops import delta as D
from slopllm_b200.ops import experts as EX
from slopllm_b200.ops import get_ops
from slopllm_b200.ops import grouped as G
from slopllm_b200.ops import latent as L
from slopllm_b200.ops import recurrent as RC
from slopllm_b200.ops.rotary import rotary_table
from zemezen_util import configs, feed, make_engine, portions, random_ids, row_error

pytestmark = pytest.mark.gpu
CONFIGS = configs()
BF16_TOL, FP32_TOL = 0.06, 3e-5      # of the logits' spread
DTYPES = [torch.float32, torch.bfloat16]


def rel(got, want):
    got, want = got.detach().double().cpu(), want.detach().double().cpu()
    return ((got - want).norm() / want.norm().clamp(min=1e-12)).item()


def gen(seed):
    return torch.Generator().manual_seed(seed)


def ops_of(dtype):
    return get_ops(types.SimpleNamespace(rms_norm_eps=1e-5), "cuda", None, dtype)


def step_state(spans, seed=0):
    """State of a step whose sequences have `n` tokens behind `start` cached ones, in shuffled pages."""
    g, ps = gen(seed), 64
    need = [-(-(s + n) // ps) for s, n in spans]
    order = torch.randperm(sum(need) + 3, generator=g).tolist()
    pt = torch.zeros(len(spans), max(need) + 1, dtype=torch.int32)
    for b in range(len(spans)):
        for j in range(need[b]):
            pt[b, j] = order.pop()
    pos = torch.tensor([st + i for st, n in spans for i in range(n)], dtype=torch.int32)
    bi = torch.tensor([b for b, (_, n) in enumerate(spans) for _ in range(n)], dtype=torch.int32)
    st = StepState(input_ids=torch.zeros(len(pos), dtype=torch.int64, device="cuda"), positions=pos.cuda(), batch_idx=bi.cuda(),
                   page_table=pt.cuda(), max_kv_len=max(a + n for a, n in spans))
    if any(n > 1 for _, n in spans):
        st.extra["spans"], st.extra["max_q"] = spans, max(n for _, n in spans)
    return st, pt, (sum(need) + 3) * ps


# ---- residual, norms, activation --------------------------------------------------------------------------------------

@pytest.mark.parametrize("H", [44, 256, 1000, 5120])
@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_and_norm(H, dtype):
    g, ops = gen(H), ops_of(dtype)
    y, r, w = torch.randn(7, H, generator=g) * 3, torch.randn(7, H, generator=g), torch.randn(H, generator=g)
    out, res = ops.post_norm(y.cuda(), r.cuda(), None, w.cuda(), 1e-3)
    assert torch.equal(res.cpu(), y + r) and out.dtype == dtype
    assert rel(out, O.norm(y + r, w, 1e-3)) < (1e-6 if dtype == torch.float32 else 3e-3)


@pytest.mark.parametrize("I,ld,ldo,at", [(36, 100, 60, 20), (13, 31, 17, 3), (1024, 4096, 2048, 512)])
@pytest.mark.parametrize("ti,to", [(torch.float32, torch.float32), (torch.float32, torch.bfloat16), (torch.bfloat16, torch.bfloat16)])
def test_activation_between_wider_rows(I, ld, ldo, at, ti, to):
    x = torch.randn(5, ld, generator=gen(I)).to(ti).cuda()
    out = torch.full((5, ldo), 7.0, dtype=to, device="cuda")
    ops_of(to).silu_mul(x[:, at:at + 2 * I], out[:, 2:2 + I] if I == 13 else out[:, 4:4 + I])
    lo = 2 if I == 13 else 4
    want = O.silu(x[:, at:at + I].float()) * x[:, at + I:at + 2 * I].float()
    assert rel(out[:, lo:lo + I], want) < (1e-6 if to == torch.float32 else 3e-3)
    rest = torch.cat([out[:, :lo], out[:, lo + I:]], 1)
    assert bool((rest == 7).all())


# ---- grouped-query attention ------------------------------------------------------------------------------------------

def attention_case(spans, heads, kv, dim, window, keep, dtype, dims=None, sink=None, own=0, plant=None, seed=0, in_f32=False):
    """Portions `spans` = [(start, n)] over rows cached by earlier steps; `own`: value size of separate values."""
    g = gen(seed)
    st, pt, slots = step_state(spans, seed)
    vdim = own or dim
    s = G.GroupedShape(heads, kv, dim, vdim, dim ** -0.5, window, keep, 1e-5, own_values=bool(own))
    T, base = len(st.positions), 1e4
    dims = dims if dims is not None else dim
    proj = torch.randn(T, heads * dim + kv * dim + (kv * vdim if own else 0), generator=g).to(dtype)
    qn, kn = torch.randn(dim, generator=g) * 0.2 + 1, torch.randn(dim, generator=g) * 0.2 + 1
    sink = torch.randn(heads, generator=g) if sink is None else torch.full((heads,), float(sink))
    kc, vc = torch.zeros(slots, kv, dim, dtype=dtype), torch.zeros(slots, kv, vdim, dtype=dtype)
    rows = [(torch.randn(a, kv, dim, generator=g).to(dtype), torch.randn(a, kv, vdim, generator=g).to(dtype)) for a, _ in spans]
    x, want, at = proj.double(), [], 0
    turn = lambda y, w, p: O.rotate(O.norm(y, w, 1e-5), p, dims, base)
    for b, (a, n) in enumerate(spans):
        here = torch.arange(a, a + n)
        q = turn(x[at:at + n, :heads * dim].view(n, heads, dim), qn, here)
        if plant is not None:
            plant(b, a, q, rows[b][0])
        for p in range(a):
            i = int(pt[b, p // 64]) * 64 + p % 64
            kc[i], vc[i] = rows[b][0][p], rows[b][1][p]
        k0 = x[at:at + n, heads * dim:(heads + kv) * dim].view(n, kv, dim)
        v0 = x[at:at + n, (heads + kv) * dim:].view(n, kv, vdim) if own else k0
        k, v = torch.cat([rows[b][0].double(), turn(k0, kn, here)]), torch.cat([rows[b][1].double(), v0])
        k, v = k.repeat_interleave(heads // kv, 1), v.repeat_interleave(heads // kv, 1)
        w = O.softmax_with_sink(torch.einsum("thd,shd->hts", q, k) * s.scale, O.visible(a + n, window, keep)[a:], sink.double())
        want.append(torch.einsum("hts,shv->thv", w, v).reshape(n, -1))
        at += n
    w = G.GroupedWeights(qn.cuda(), kn.cuda(), sink.cuda())
    kg, vg, pg = kc.cuda(), vc.cuda(), (proj.float() if in_f32 else proj).cuda()
    q = G.grouped_pre(pg, s, w, rotary_table(dims, base).to("cuda"), st, kg, vg, dtype)
    wide = torch.full((T, heads * vdim + 8), 5.0, dtype=dtype, device="cuda")
    G.grouped_attention(q, s, w, st, kg, vg, wide[:, :heads * vdim])
    assert bool((wide[:, heads * vdim:] == 5).all())
    return wide[:, :heads * vdim], torch.cat(want)


SHAPES = [(4, 2, 16), (6, 2, 40), (3, 3, 128), (20, 1, 64), (16, 2, 96), (2, 1, 256), (4, 2, 12), (1, 1, 8), (2, 2, 56), (3, 1, 104)]
SPANS = [[(0, 130), (70, 3), (200, 1), (5, 64)], [(150, 1), (3, 1), (0, 1), (256, 1)], [(127, 2)], [(0, 1)], [(300, 40)]]


@pytest.mark.parametrize("heads,kv,dim", SHAPES)
@pytest.mark.parametrize("window,keep", [(1, 1), (9, 3), (64, 64), (65, 5), (100, 70), (0, 0), (33, 0), (33, 128)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_grouped_attention(heads, kv, dim, window, keep, dtype):
    for spans in SPANS:
        got, want = attention_case(spans, heads, kv, dim, window, keep, dtype)
        assert rel(got, want) < (2e-5 if dtype == torch.float32 else 1.2e-2), spans


@pytest.mark.parametrize("dtype", DTYPES)
def test_grouped_attention_partial_rotation_own_values_fp32_rows(dtype):
    tol = 2e-5 if dtype == torch.float32 else 1.2e-2
    for spans in SPANS:
        for kw in (dict(dims=8), dict(dims=2), dict(own=24), dict(own=8, dims=16), dict(in_f32=True)):
            got, want = attention_case(spans, 6, 2, 32, 50, 4, dtype, **kw)
            assert rel(got, want) < tol, (spans, kw)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,keep", [(2, 1), (40, 5), (64, 64), (65, 6), (128, 7), (129, 65), (300, 4)])
@pytest.mark.parametrize("place", ["window_in", "window_out", "first_in", "first_out"])
def test_one_key_at_an_edge(window, keep, place, dtype):
    """One cached key answers the query far better than all others and sits on the last position that the window shows, just
    outside it, on the last kept token or on the one behind it.  Decoded rows and the first row of portions, around page borders."""
    def at(start):
        return {"window_in": start - window + 1, "window_out": start - window, "first_in": keep - 1, "first_out": keep}[place]

    def plant(b, start, q, keys):
        keys[at(start)] = (q[0].mean(0, keepdim=True) * 12.0).to(keys.dtype).expand_as(keys[0])

    low = window + keep + 1                                       # (the kept tokens and the window do not touch)
    for spans in ([(s, 1) for s in sorted({low, 447, 448, 449, 511, 512})], [(low, 2), (449, 2), (512, 130)]):
        got, want = attention_case(spans, 1, 1, 16, window, keep, dtype, sink=0.0, plant=plant, seed=window)
        row = 0
        for s, n in spans:
            assert rel(got[row], want[row]) < (2e-5 if dtype == torch.float32 else 1.5e-2), (s, n)
            row += n
        wrong = {"window_in": (window - 1, keep), "window_out": (window + 1, keep), "first_in": (window, keep - 1), "first_out": (window, keep + 1)}[place]
        if wrong[0] > 0:                                          # the planted key decides the row
            _, other = attention_case(spans, 1, 1, 16, *wrong, dtype, sink=0.0, plant=plant, seed=window)
            assert rel(other[0], want[0]) > 0.2


@pytest.mark.parametrize("sink", [-30.0, 0.0, 7.0])
@pytest.mark.parametrize("dtype", DTYPES)
def test_sink_mass(sink, dtype):
    tol = 2e-5 if dtype == torch.float32 else 1.2e-2
    for spans in ([(100, 1), (30, 40)], [(1500, 1), (3, 1)]):
        got, want = attention_case(spans, 4, 2, 16, 900, 3, dtype, sink=sink)
        assert rel(got, want) < tol
        none, _ = attention_case(spans, 4, 2, 16, 900, 3, dtype, sink=-1e4)
        assert (rel(got, none) < 1e-6) == (sink == -30.0)


def test_decode_key_splits():
    """Long contexts: the keys of one row are shared by several blocks, the sink counts once."""
    for spans, window, keep in (([(1500, 1), (700, 1)], 600, 70), ([(1999, 1)], 0, 0), ([(64 * i + 5, 1) for i in range(40)], 333, 4)):
        got, want = attention_case(spans, 8, 2, 64, window, keep, torch.bfloat16, sink=3.0)
        assert rel(got, want) < 1.2e-2


# ---- latent attention without positions ---------------------------------------------------------------------------------

@pytest.mark.parametrize("heads,dim,vdim,rank", [(3, 16, 24, 40), (2, 128, 128, 512), (5, 40, 88, 64), (2, 24, 136, 264), (3, 12, 20, 36), (17, 64, 32, 128)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_attention(heads, dim, vdim, rank, dtype):
    for spans in SPANS + [[(1500, 1), (64, 1)]]:
        g = gen(rank)
        st, pt, slots = step_state(spans)
        s = L.LatentShape(heads, dim, 0, vdim, rank, dim ** -0.5, 0, 1e-5)
        T = len(st.positions)
        qd, norm = torch.randn(T, heads * dim + rank, generator=g).to(dtype), torch.randn(rank, generator=g)
        uk, uv = ((torch.randn(heads, d, rank, generator=g) * rank ** -0.5).to(dtype) for d in (dim, vdim))
        cache = torch.zeros(slots, rank, dtype=dtype)
        want, at = [], 0
        for b, (a, n) in enumerate(spans):
            old = torch.randn(a, rank, generator=g).to(dtype)
            for p in range(a):
                cache[int(pt[b, p // 64]) * 64 + p % 64] = old[p]
            x = qd[at:at + n].double()
            c = torch.cat([old.double(), O.norm(x[:, heads * dim:], norm, 1e-5)])
            k, v = (torch.einsum("hdr,sr->shd", u.double(), c) for u in (uk, uv))
            w = O.softmax_with_sink(torch.einsum("thd,shd->hts", x[:, :heads * dim].view(n, heads, dim), k) * s.scale, O.visible(a + n)[a:])
            want.append(torch.einsum("hts,shv->thv", w, v).reshape(n, -1))
            at += n
        w = L.LatentWeights(norm.cuda(), uk.cuda(), uv.cuda(), uv.transpose(1, 2).contiguous().cuda())
        cg, qg = cache.cuda(), qd.cuda()
        q_rot = L.latent_pre(qg, s, w, rotary_table(0, 1.0).to("cuda"), st, cg)
        wide = torch.full((T, heads * vdim + 8), 5.0, dtype=dtype, device="cuda")
        got = L.latent_attention(qg, q_rot, s, w, st, cg, ops_of(dtype), wide[:, :heads * vdim])
        assert bool((wide[:, heads * vdim:] == 5).all())
        assert rel(got, torch.cat(want)) < (2e-5 if dtype == torch.float32 else 1.2e-2), spans


# ---- gated delta rule ---------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
@pytest.mark.parametrize("dtype", DTYPES)
def test_short_convolution(taps, dtype):
    """Sequences in portions of every size, their histories in rings of reused, shuffled slots."""
    g, Cn = gen(taps), 150
    total = [90, 41, 7, 1]
    x = [torch.randn(n, Cn, generator=g).to(dtype) for n in total]
    w = torch.randn(Cn, taps, generator=g)
    want = [O.short_conv(y.double(), w) for y in x]
    state = torch.zeros(6, taps, Cn, device="cuda")
    slots, done, got = [4, 0, 5, 2], [0] * 4, [[] for _ in total]
    for cut in ([40, 1, 2, 1], [1, 1, 1, 0], [2, 33, 3, 0], [33, 2, 1, 0], [1, 4, 0, 0], [13, 0, 0, 0]):
        live = [b for b in range(4) if cut[b]]
        ind = torch.tensor([0] + [cut[b] for b in live]).cumsum(0).to(torch.int32)
        pos = torch.cat([torch.arange(done[b], done[b] + cut[b]) for b in live]).to(torch.int32)
        rows = torch.cat([x[b][done[b]:done[b] + cut[b]] for b in live])
        wide = torch.zeros(len(rows), Cn + 6, dtype=dtype)
        wide[:, :Cn] = rows
        y = D.short_conv(wide.cuda()[:, :Cn], w.t().contiguous().cuda(), state, pos.cuda(), ind.cuda(), torch.tensor([slots[b] for b in live], dtype=torch.int32).cuda(),
                         max(cut), dtype).cpu()
        for j, b in enumerate(live):
            got[b].append(y[ind[j]:ind[j + 1]])
            done[b] += cut[b]
    assert done == total
    for b in range(4):
        assert rel(torch.cat(got[b]), want[b]) < (1e-6 if dtype == torch.float32 else 3e-3)


def delta_case(lens, h, hk, dk, dv, taps, dtype, rate=0.0, bias=-3.0, seed=0, fresh=False, gain=1.0):
    """Portions behind `start` earlier tokens from a non-zero state; returns (arguments of the op, wanted output, wanted state)."""
    g = gen(seed)
    T, B, ra, rg = sum(lens), len(lens), 8, 16
    s = D.DeltaShape(h, hk, dk, dv, taps, 1e-4)
    start = [0 if fresh else 5 + 3 * b for b in range(B)]
    r = lambda *n: torch.randn(*n, generator=g)
    main, fine = (r(T, s.channels) * gain).to(dtype), r(T, ra + rg + h)
    conv = r(s.channels, taps) * taps ** -0.5
    a2, g2 = (r(h * dk, ra) * ra ** -0.5).to(dtype), (r(h * dv, rg) * rg ** -0.5).to(dtype)
    dt, A_log, nw = r(h * dk) + bias, r(h) * 0.5 + rate, r(dv)
    slots = [(2 * b + 1) % (B + 2) for b in range(B)] if (B + 2) % 2 else list(range(B))[::-1]
    S, ring = torch.zeros(B + 2, h, dk, dv), torch.zeros(B + 2, taps, s.channels)
    want, at, S_want = [], 0, {}
    if dtype == torch.bfloat16 and max(lens) >= RC.CHUNK_MIN_Q:
        low = fine[:, :ra + rg].bfloat16().double()               # (operands of a product there)
    else:
        low = fine[:, :ra + rg].double()
    for b, n in enumerate(lens):
        hist = r(start[b], s.channels).to(dtype)
        for p in range(max(0, start[b] - taps), start[b]):
            ring[slots[b], p % taps] = hist[p].float()
        if not fresh:
            S[slots[b]] = r(h, dk, dv)
        x = O.short_conv(torch.cat([hist, main[at:at + n]]).double(), conv)[start[b]:]
        if dtype == torch.bfloat16 and max(lens) > 1:
            x = x.bfloat16().double()
        qk = hk * dk
        grow = lambda y: O.unit(y.view(n, hk, dk)).repeat_interleave(h // hk, 1)
        q, k, v = grow(x[:, :qk]) * dk ** -0.5, grow(x[:, qk:2 * qk]), x[:, 2 * qk:].view(n, h, dv)
        f = low[at:at + n]
        decay = torch.exp(-torch.exp(A_log.double())[:, None] * O.softplus(f[:, :ra] @ a2.double().t() + dt.double()).view(n, h, dk))
        beta = torch.sigmoid(fine[at:at + n, ra + rg:].double())
        st, o = S[slots[b]].double(), []
        for i in range(n):
            st = decay[i][:, :, None] * st
            u = beta[i][:, None] * (v[i] - (st * k[i][:, :, None]).sum(1))
            st = st + k[i][:, :, None] * u[:, None, :]
            o.append((st * q[i][:, :, None]).sum(1))
        S_want[slots[b]] = st
        o = O.rms(torch.stack(o), s.eps) * nw.double()
        want.append(o.reshape(n, -1) * torch.sigmoid(f[:, ra:] @ g2.double().t()))
        at += n
    w = D.DeltaWeights(conv.t().contiguous().cuda(), a2.cuda(), g2.cuda(), dt.cuda(), A_log.cuda(), nw.cuda())
    ind = torch.tensor([0] + lens).cumsum(0).to(torch.int32).cuda()
    st = types.SimpleNamespace(positions=torch.cat([torch.arange(a, a + n) for a, n in zip(start, lens)]).to(torch.int32).cuda(), extra={})
    if max(lens) > 1:
        st.extra = {"spans": list(zip(start, lens)), "max_q": max(lens)}
    args = (main.cuda(), fine.cuda(), s, w, S.cuda(), ring.cuda(), st, ind, torch.tensor(slots, dtype=torch.int32).cuda())
    return args, torch.cat(want), S_want


def run_delta(args, dtype, plan):
    main, fine, s, w, S, ring, st, ind, slots = args
    S, ring = S.clone(), ring.clone()
    wide = torch.full((main.shape[0], s.heads * s.dv + 8), 5.0, dtype=dtype, device="cuda")
    D.channel_delta_mix(main, fine, s, w, S, ring, st, ind, slots, wide[:, :s.heads * s.dv], ops_of(dtype), plan)
    assert bool((wide[:, s.heads * s.dv:] == 5).all())
    return wide[:, :s.heads * s.dv], S


DELTAS = [([200, 1, 64, 17], 2, 2, 32, 48, 4), ([130], 3, 1, 128, 128, 4), ([65, 63, 3], 4, 2, 40, 24, 3), ([33, 2], 2, 1, 10, 7, 2),
          ([70], 2, 2, 24, 160, 1), ([1, 1, 1], 4, 2, 64, 32, 4), ([1, 1], 2, 2, 9, 13, 3), ([1], 2, 1, 128, 128, 2), ([129], 2, 1, 136, 96, 2),
          ([1], 1, 1, 200, 264, 2), ([192, 128], 2, 2, 16, 8, 5)]


@pytest.mark.parametrize("lens,h,hk,dk,dv,taps", DELTAS)
@pytest.mark.parametrize("rate,bias", [(0.0, -3.0), (2.0, 2.0), (-3.0, -6.0)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_channel_delta(lens, h, hk, dk, dv, taps, rate, bias, dtype):
    """Decays between nearly none and everything within a token; from non-zero states and convolution histories."""
    args, want, S_want = delta_case(lens, h, hk, dk, dv, taps, dtype, rate, bias, seed=dk)
    plans = [None] + ([RC.ChunkPlan(lens, "cuda")] if dtype == torch.bfloat16 and max(lens) >= RC.CHUNK_MIN_Q else [])
    for plan in plans:
        got, S = run_delta(args, dtype, plan)
        for slot, x in S_want.items():
            assert rel(S[slot], x) < (1e-5 if dtype == torch.float32 else 4e-3), plan
        assert rel(got, want) < (2e-5 if dtype == torch.float32 else 8e-3), plan


@pytest.mark.parametrize("dk,dv", [(128, 128), (48, 80), (144, 72)])
def test_chunks_keep_fp32_accuracy(dk, dv):
    """Repeated keys and weak decay make the triangular system of a chunk ill-conditioned in 16 bits; the chunked state follows the
    token-by-token kernel far below bf16 rounding (both start from the same convolved rows)."""
    args, _, _ = delta_case([200, 90], 2, 1, dk, dv, 1, torch.bfloat16, rate=-2.0, bias=-5.0, seed=3, fresh=True)
    main = args[0]
    main[:, dk:2 * dk] = main[:1, dk:2 * dk] + 0.1 * main[:, dk:2 * dk]          # the key channels hardly change
    main[:, :2 * dk] = main[:, :2 * dk].abs() + 0.5
    fine = args[1]
    fine[:, :24] = fine[:, :24].bfloat16().float()
    a, S = run_delta(args, torch.bfloat16, None)
    b, Sc = run_delta(args, torch.bfloat16, RC.ChunkPlan([200, 90], "cuda"))
    assert rel(Sc, S) < 5e-5 and rel(b, a) < 4e-3


def test_chunk_passes_carry_the_state(monkeypatch):
    """Scratch for two chunks only: the passes of one step hand the state on."""
    from slopllm_b200.ops import delta_chunk as DC
    args, _, _ = delta_case([300, 90], 2, 1, 32, 40, 4, torch.bfloat16, seed=5)
    out = []
    for budget in (256 << 20, 2 * 2 * DC.scratch_bytes(32, 40)):
        monkeypatch.setattr(DC, "SCRATCH_BYTES", budget)
        out.append(run_delta(args, torch.bfloat16, RC.ChunkPlan([300, 90], "cuda")))
    for a, b in zip(*out):
        assert rel(a, b) < 1e-5


def test_a_lost_term_shows():
    """The cases above mean something only if small mistakes move the result."""
    args, want, _ = delta_case([70], 2, 1, 32, 48, 4, torch.float32)
    main, fine, s, w, S, ring, st, ind, slots = args
    for change in ("beta", "decay", "history", "gate", "norm"):
        f, wc, r = fine.clone(), w, ring.clone()
        if change == "beta":
            f[:, 24:] += 0.3
        elif change == "decay":
            f[:, :8] = f[:, :8].roll(1, 0)
        elif change == "history":
            r.zero_()
        elif change == "gate":
            f[:, 8:24] = 0
        else:
            wc = D.DeltaWeights(w.conv, w.a2, w.g2, w.dt_bias, w.A_log, torch.ones_like(w.norm))
        got, _ = run_delta((main, f, s, wc, S, r, st, ind, slots), torch.float32, None)
        assert rel(got, want) > 5e-3, change


# ---- routed experts -----------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("E,top,groups,keep", [(15, 4, 5, 3), (1, 1, 1, 1), (40, 6, 8, 3), (9, 4, 3, 2), (64, 8, 1, 1), (256, 8, 8, 4), (300, 5, 100, 2), (1000, 16, 10, 10)])
def test_routing(E, top, groups, keep):
    g = gen(E)
    z = torch.randn(37, E + 3, generator=g) * 2
    ids, w = EX.route_softmax(z.cuda()[:, :E], top, groups, keep)
    dense = torch.zeros(37, E).scatter(1, ids.long().cpu(), w.cpu())
    assert rel(dense, O.choose_experts(z[:, :E].double(), top, groups, keep)) < 1e-6
    assert all(len(set(r)) == top for r in ids.tolist())
    if groups > 1:                                                # one high score opens a group of otherwise low ones
        z[:, :E] = 0
        z[:, E - 1], z[:, :E // groups] = 5.0, 1.0
        ids, w = EX.route_softmax(z.cuda()[:, :E], top, groups, 1) if top <= E // groups else EX.route_softmax(z.cuda()[:, :E], top, groups, keep)
        assert bool((ids[:, 0] == E - 1).all())


@pytest.mark.parametrize("T", [1, 2, 9, 32, 33, 200])
@pytest.mark.parametrize("E,top,H,I", [(11, 3, 64, 32), (4, 2, 256, 64), (5, 5, 44, 12), (40, 6, 128, 48), (16, 4, 1024, 256)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_experts(T, E, top, H, I, dtype):
    g = gen(T + E)
    x = torch.randn(T, H, generator=g).to(dtype)
    w13, w2 = (torch.randn(E, 2 * I, H, generator=g) * H ** -0.5).to(dtype), (torch.randn(E, H, I, generator=g) * I ** -0.5).to(dtype)
    z = torch.randn(T, E, generator=g)
    z[:, 0] += 3                                                  # one expert that many tokens share
    w = O.choose_experts(z.double(), top)
    base = torch.randn(T, H, generator=g)
    want = base.double()
    for e in range(E):
        a = x.double() @ w13[e].double().t()
        want += w[:, e, None] * ((O.silu(a[:, :I]) * a[:, I:]) @ w2[e].double().t())
    ids = w.topk(top, -1).indices.to(torch.int32)
    out = base.cuda()
    EX.add_experts(x.cuda(), ExpertWeights(w13.cuda(), w2.cuda()), ids.cuda(), w.gather(1, ids.long()).float().cuda(), out, ops_of(dtype))
    assert rel(out, want) < (1e-5 if dtype == torch.float32 else 6e-3)


# ---- whole models through the engine ----------------------------------------------------------------------------------

@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", DTYPES)
def test_engine_schedules(name, dtype):
    """Whole prompt, portions down to two tokens, token by token: all positions against the plain forward."""
    raw, ranks = CONFIGS[name]
    t = O.random_tensors(raw, 1, ranks)
    ids = random_ids(raw, 200, 2)
    want = O.forward(raw, t, ids)
    eng = make_engine(raw, t, "cuda", dtype)
    for cuts in ([200], portions(200, [2, 64, 3, 29, 70]), portions(200, [150], tail=40), [1] * 200):
        err = row_error(feed(eng, ids, cuts), want)
        if dtype == torch.float32:
            assert err.max() < FP32_TOL, (cuts[:5], err.argmax(), err.max())
        else:                                                     # (a close call of the router moves single positions)
            assert err.mean() < BF16_TOL / 2 and (err > 2 * BF16_TOL).float().mean() < 0.03, (cuts[:5], err.argmax(), err.max())


@pytest.mark.parametrize("dtype", DTYPES)
def test_engine_mixed_batches_and_reused_slots(dtype):
    raw, ranks = CONFIGS["tiled"]
    t = O.random_tensors(raw, 3, ranks)
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
        assert err.mean() < (FP32_TOL if dtype == torch.float32 else BF16_TOL / 2), (i, err.mean())
        assert (err > (FP32_TOL if dtype == torch.float32 else 2 * BF16_TOL)).float().mean() < (1e-9 if dtype == torch.float32 else 0.05), (i, err.max())


def far_key_model():
    """Nearly undamped recurrences and sharp attention, so that tokens hundreds of positions back stay in the logits."""
    raw, ranks = CONFIGS["tiled"]
    t = O.random_tensors(raw, 4, ranks)
    for i in (1, 3):
        t[f"l{i}.mix.dt_bias"] = t[f"l{i}.mix.dt_bias"] - 5
    t["l2.mix.q"] = t["l2.mix.q"] * 3
    return raw, t


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    """Hundreds of decoded tokens over page borders and through the window, in a graph."""
    raw, t = far_key_model()
    ids = random_ids(raw, 420, 6)
    want = O.forward(raw, t, ids)
    changed = O.forward(raw, t, [(ids[0] + 1) % raw["vocab"]] + ids[1:])
    assert row_error(changed, want)[-1] > 0.02                    # the first token still matters at the end
    err = row_error(feed(make_engine(raw, t, "cuda", dtype), ids, [60] + [1] * 360), want)
    assert err.mean() < (5e-5 if dtype == torch.float32 else BF16_TOL), err.mean()
    assert (err > (2e-4 if dtype == torch.float32 else 3 * BF16_TOL)).float().mean() < 0.03, (err.argmax(), err.max())


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_scheduler(dtype):
    from slopllm_b200.config import SamplingParams
    from slopllm_b200.sampling.workspace import SamplingWorkspace
    from slopllm_b200.scheduler.scheduler import GenerationRequest, GenerationScheduler
    raw, ranks = CONFIGS["wide"]
    t = O.random_tensors(raw, 7, ranks)
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
