"""Gidisun's sm_100a kernels: every mechanism alone and whole models through the engine, against the plain implementation."""
import types

import pytest
import torch

import gidisun_oracle as O
from gidisun_util import YARN, configs, feed, make_engine, portions, random_ids, row_error
from slopllm_b200.models.glm_moe_dsa import StepState
from slopllm_b200.ops import get_ops
from slopllm_b200.ops import latent as L
from slopllm_b200.ops import recurrent as RC
from slopllm_b200.ops.rotary import YarnScaling, rotary_table

pytestmark = pytest.mark.gpu
CONFIGS = configs()
BF16_TOL, FP32_TOL = 0.06, 3e-5      # of the logits' spread; bf16 rounding of these models stays below 0.03


def rel(got, want):
    got, want = got.detach().float().cpu(), want.detach().float().cpu()
    return ((got - want).norm() / want.norm().clamp(min=1e-12)).item()


def gen(seed):
    return torch.Generator().manual_seed(seed)


# ---- mechanisms -----------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("H", [44, 256, 1000, 5120])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_sandwich_norms(H, dtype):
    g = gen(H)
    ops = get_ops(types.SimpleNamespace(rms_norm_eps=1e-5), "cuda", None, dtype)
    y, r, wp, wn = torch.randn(7, H, generator=g) * 3, torch.randn(7, H, generator=g), torch.randn(H, generator=g), torch.randn(H, generator=g)
    out, res = ops.post_norm(y.cuda(), r.cuda(), (1 + wp).cuda(), (1 + wn).cuda(), 1e-3)
    want = r + O.norm_around_zero(y, wp, 1e-3)
    assert out.dtype == dtype and rel(res, want) < 1e-6
    assert rel(out, O.norm_around_zero(want, wn, 1e-3)) < (1e-6 if dtype == torch.float32 else 3e-3)
    table = torch.randn(11, H, generator=g).to(dtype)
    ids = torch.tensor([0, 10, 3])
    out, res = ops.embed_norm(ids.cuda(), table.cuda(), (1 + wn).cuda(), 1e-3)
    assert torch.equal(res.cpu(), table[ids].float()) and rel(out, O.norm_around_zero(table[ids].float(), wn, 1e-3)) < 3e-3


@pytest.mark.parametrize("T,N,K,heads", [(1, 5, 7, 1), (70, 130, 33, 3), (3, 64, 100, 2)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_products_of_any_shape(T, N, K, heads, dtype):
    g = gen(T)
    ops = get_ops(types.SimpleNamespace(rms_norm_eps=1e-5), "cuda", None, dtype)
    from slopllm_b200.models.weights import LinearWeight
    x, w = torch.randn(T, K, generator=g).to(dtype), torch.randn(N, K, generator=g).to(dtype)
    want = x.double() @ w.double().t()
    assert rel(ops.linear(x.cuda(), LinearWeight(w.cuda()), out_f32=True), want) < 1e-5
    xh, wh = torch.randn(T, heads * (K + 2), generator=g).to(dtype), torch.randn(heads, K, N, generator=g).to(dtype)
    want = torch.einsum("thk,hkn->thn", xh.double().view(T, heads, K + 2)[..., :K], wh.double()).reshape(T, -1)
    assert rel(L.head_product(xh.cuda(), K + 2, wh.cuda(), ops), want) < (1e-5 if dtype == torch.float32 else 4e-3)


def scan_inputs(lens, h, dk, dv, seed, dtype):
    g = gen(seed)
    T, B = sum(lens), len(lens)
    x = types.SimpleNamespace(T=T, B=B, h=h, dk=dk, dv=dv, lens=lens)
    x.proj = torch.randn(T, h * 2 * (dk + dv), generator=g).to(dtype)
    x.S, x.n, x.m = torch.randn(B + 2, h, dk, dv, generator=g), torch.randn(B + 2, h, dk, generator=g), torch.randn(B + 2, h, generator=g) * 2
    x.ind = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32)
    x.slots = torch.tensor([(3 * b + 1) % (B + 2) for b in range(B)] if (B + 2) % 3 else list(range(B))[::-1], dtype=torch.int32)
    x.parts = [t.float() for t in torch.split(x.proj, [h * dk, h * dk, h * dv, h * dv], 1)]
    x.g = g
    return x


def split(x, lo, hi):
    q, k, v, g = (p[lo:hi].view(hi - lo, x.h, -1) for p in x.parts)
    return q * x.dk ** -0.5, k, v, g


SCANS = [([200, 1, 64, 17], 2, 32, 48), ([130], 3, 128, 128), ([65, 63, 3], 1, 40, 24), ([33, 2], 2, 10, 7), ([70], 2, 24, 160),
         ([1, 1, 1], 4, 64, 32), ([1, 1], 2, 9, 13)]


def forms(lens, dtype):
    """The chunked kernels (portions of bf16 models) and the step kernel."""
    return [None] + ([RC.ChunkPlan(lens, "cuda")] if dtype == torch.bfloat16 and max(lens) > 1 else [])


@pytest.mark.parametrize("lens,h,dk,dv", SCANS)
@pytest.mark.parametrize("dtype,tau,shift", [(torch.bfloat16, 16.0, 2.0), (torch.bfloat16, 1.0, -8.0), (torch.float32, 3.0, 0.0)])
def test_gla(lens, h, dk, dv, dtype, tau, shift):
    """From a non-zero state; `shift` moves the decays between close to one and close to zero within a token."""
    x = scan_inputs(lens, h, dk, dv, 1, dtype)
    rank = 6
    low, a2, a2b = torch.randn(x.T, rank, generator=x.g), torch.randn(h * dk, rank, generator=x.g).to(dtype), torch.randn(h * dk, generator=x.g) + shift
    nw = torch.randn(dv, generator=x.g)
    alpha = torch.sigmoid((low @ a2.float().t() + a2b).double()).pow(1.0 / tau).view(x.T, h, dk)
    want, S = torch.empty(x.T, h, dv, dtype=torch.float64), x.S.double()
    for b in range(x.B):
        lo, hi, slot = int(x.ind[b]), int(x.ind[b + 1]), int(x.slots[b])
        q, k, v, g = (p.double() for p in split(x, lo, hi))
        for i in range(hi - lo):
            S[slot] = alpha[lo + i][:, :, None] * S[slot] + k[i][:, :, None] * v[i][:, None, :]
            want[lo + i] = (S[slot] * q[i][:, :, None]).sum(1)
        want[lo:hi] = O.rms(want[lo:hi], 1e-4) * nw.double() * O.silu(g)
    for plan in forms(lens, dtype):
        Sg = x.S.cuda()
        got = RC.gla_mix(x.proj.cuda(), low.cuda(), a2.cuda(), a2b.cuda(), tau, nw.cuda(), 1e-4, Sg, x.ind.cuda(), x.slots.cuda(), h, dk, dv, dtype, plan)
        assert rel(Sg, S) < 1e-5, plan
        assert rel(got, want.reshape(x.T, -1)) < (1e-5 if dtype == torch.float32 else 3e-3), plan


@pytest.mark.parametrize("lens,h,dk,dv", SCANS)
@pytest.mark.parametrize("dtype,cap,shift", [(torch.bfloat16, 12.0, -2.0), (torch.bfloat16, 30.0, 20.0), (torch.float32, 5.0, 0.0)])
def test_mlstm(lens, h, dk, dv, dtype, cap, shift):
    x = scan_inputs(lens, h, dk, dv, 2, dtype)
    gates, ib, fb = torch.randn(x.T, 2 * h, generator=x.g) * 3, torch.randn(h, generator=x.g) + shift, torch.randn(h, generator=x.g) + 3
    nw = torch.randn(h * dv, generator=x.g)
    gi = cap * torch.tanh((gates[:, :h].double() + ib) / cap)
    gf = torch.nn.functional.logsigmoid(cap * torch.tanh((gates[:, h:].double() + fb) / cap))
    want, S, n, m = torch.empty(x.T, h, dv, dtype=torch.float64), x.S.double(), x.n.double(), x.m.double()
    for b in range(x.B):
        lo, hi, s = int(x.ind[b]), int(x.ind[b + 1]), int(x.slots[b])
        q, k, v, g = (p.double() for p in split(x, lo, hi))
        for i in range(hi - lo):
            top = torch.maximum(gf[lo + i] + m[s], gi[lo + i])
            keep, add = torch.exp(gf[lo + i] + m[s] - top), torch.exp(gi[lo + i] - top)
            S[s] = keep[:, None, None] * S[s] + add[:, None, None] * k[i][:, :, None] * v[i][:, None, :]
            n[s] = keep[:, None] * n[s] + add[:, None] * k[i]
            m[s] = top
            den = torch.maximum((n[s] * q[i]).sum(-1).abs(), torch.exp(-m[s])) + 1e-6
            want[lo + i] = (S[s] * q[i][:, :, None]).sum(1) / den[:, None]
        want[lo:hi] = O.rms(want[lo:hi], 1e-4) * nw.double().view(h, dv) * torch.sigmoid(g)
    for plan in forms(lens, dtype):
        state = (x.S.cuda(), x.n.cuda(), x.m.cuda())
        got = RC.mlstm_mix(x.proj.cuda(), gates.cuda(), ib.cuda(), fb.cuda(), cap, nw.cuda(), 1e-4, state, x.ind.cuda(), x.slots.cuda(), h, dk, dv,
                           dtype, plan)
        for a, w in zip(state, (S, n, m)):
            assert rel(a, w) < 1e-5, plan
        assert rel(got, want.reshape(x.T, -1)) < (3e-5 if dtype == torch.float32 else 3e-3), plan


def test_chunk_passes_carry_the_state(monkeypatch):
    """Scratch for two chunks only: the passes of one step hand the state on."""
    x = scan_inputs([300, 90], 2, 32, 40, 5, torch.bfloat16)
    gates, ib, fb, nw = (t.cuda() for t in (torch.randn(x.T, 4, generator=x.g), torch.randn(2, generator=x.g), torch.randn(2, generator=x.g) + 3,
                                            torch.randn(80, generator=x.g)))
    out = []
    for budget in (96 << 20, 2 * 2 * 32 * 40 * 4):
        monkeypatch.setattr(RC, "CHUNK_SCRATCH_BYTES", budget)
        state = (x.S.cuda(), x.n.cuda(), x.m.cuda())
        o = RC.mlstm_mix(x.proj.cuda(), gates, ib, fb, 9.0, nw, 1e-5, state, x.ind.cuda(), x.slots.cuda(), 2, 32, 40, torch.bfloat16,
                         RC.ChunkPlan(x.lens, "cuda"))
        out.append((o, *state))
    for a, b in zip(*out):
        assert rel(a, b) < 1e-5


def attention_case(spans, heads, dim, rot_dim, vdim, rank, window, dtype, sink=None, dims=None, plant=None, seed=0):
    """Latent attention of portions `spans` = [(start, n)] whose earlier rows lie in shuffled pages, and the same computed
    plainly.  `plant(spans, query tokens q_rot-part, key rows by (sequence, position))` may sharpen chosen scores."""
    g = gen(seed)
    B, ps, D = len(spans), 64, dim + rot_dim
    need = [-(-(s + n) // ps) for s, n in spans]
    order = torch.randperm(sum(need) + 3, generator=g).tolist()
    pt = torch.zeros(B, max(need) + 1, dtype=torch.int32)
    for b in range(B):
        for j in range(need[b]):
            pt[b, j] = order.pop()
    s = L.LatentShape(heads, dim, rot_dim, vdim, rank, D ** -0.5, window, 1e-5)
    rot = {"dims": dims or rot_dim, "base": 1e4, "scaling": YARN}
    T = sum(n for _, n in spans)
    qd = (torch.randn(T, heads * D + s.row, generator=g)).to(dtype)
    norm = torch.randn(rank, generator=g)
    uk, uv = ((torch.randn(heads, d, rank, generator=g) * rank ** -0.5).to(dtype) for d in (dim, vdim))
    sink = torch.randn(heads, generator=g) if sink is None else torch.full((heads,), float(sink))
    cache = torch.zeros((sum(need) + 3) * ps, s.row, dtype=dtype)
    rows = [torch.randn(st, s.row, generator=g).to(dtype) for st, _ in spans]        # rows cached by earlier steps
    if plant is not None:
        plant(spans, qd, rows, s, rot)
    pos = torch.tensor([st + i for st, n in spans for i in range(n)], dtype=torch.int32)
    bi = torch.tensor([b for b, (_, n) in enumerate(spans) for _ in range(n)], dtype=torch.int32)
    want, at = [], 0
    for b, (st, n) in enumerate(spans):
        for p in range(st):
            cache[int(pt[b, p // ps]) * ps + p % ps] = rows[b][p]
        x = qd[at:at + n].double()
        q = x[:, :heads * D].view(n, heads, D)
        lat = O.rms(x[:, heads * D:heads * D + rank], 1e-5) * norm.double()
        here = torch.arange(st, st + n)
        keys = torch.cat([rows[b].double(), torch.cat([lat, O.rotate_half(x[:, heads * D + rank:], here, rot)], 1)])
        q_rot = O.rotate_half(q[..., dim:], here, rot)
        k, v = (torch.einsum("hdr,sr->hsd", u.double(), keys[:, :rank]) for u in (uk, uv))
        sc = torch.einsum("thd,hsd->hts", q[..., :dim], k) + torch.einsum("thd,sd->hts", q_rot, keys[:, rank:])
        w = O.sink_softmax(sc * s.scale, O.window_mask(st + n, window)[st:], sink.double())
        want.append(torch.einsum("hts,hsv->thv", w, v).reshape(n, -1))
        at += n
    st = StepState(input_ids=torch.zeros(T, dtype=torch.int64, device="cuda"), positions=pos.cuda(), batch_idx=bi.cuda(), page_table=pt.cuda(),
                   max_kv_len=max(a + n for a, n in spans))
    if any(n > 1 for _, n in spans):
        st.extra["spans"] = spans
    w = L.LatentWeights(norm.cuda(), uk.cuda(), uv.cuda(), uv.transpose(1, 2).contiguous().cuda(), sink.cuda())
    table = rotary_table(rot["dims"], 1e4, YarnScaling(**YARN)).to("cuda")
    ops = get_ops(types.SimpleNamespace(rms_norm_eps=1e-5), "cuda", None, dtype)
    cg, qg = cache.cuda(), qd.cuda()
    q_rot = L.latent_pre(qg, s, w, table, st, cg)
    return L.latent_attention(qg, q_rot, s, w, st, cg, ops), torch.cat(want)


ATTN = [(3, 16, 8, 24, 40), (2, 128, 64, 128, 512), (5, 32, 16, 48, 64), (2, 24, 16, 136, 264), (3, 12, 10, 20, 36), (17, 16, 16, 16, 64)]


@pytest.mark.parametrize("heads,dim,rot_dim,vdim,rank", ATTN)
@pytest.mark.parametrize("window", [1, 9, 64, 65, 200, 0])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_latent_attention(heads, dim, rot_dim, vdim, rank, window, dtype):
    tol = 2e-5 if dtype == torch.float32 else 1.2e-2
    for spans in ([(0, 130), (70, 3), (200, 1), (5, 64)], [(150, 1), (3, 1), (0, 1), (256, 1)], [(127, 2)]):
        got, want = attention_case(spans, heads, dim, rot_dim, vdim, rank, window, dtype)
        assert rel(got, want) < tol, spans
    got, want = attention_case([(40, 33), (90, 1)], heads, dim, rot_dim, vdim, rank, window, dtype, sink=5.0, dims=2 * (rot_dim // 4))
    assert rel(got, want) < tol


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window", [2, 40, 64, 65, 128, 129, 300])
@pytest.mark.parametrize("inside", [True, False])
def test_one_key_at_the_window_edge(window, inside, dtype):
    """One cached key answers the query far better than all others and sits on the last position the window shows, or just
    outside it; the plain softmax then is nearly one-hot, or knows nothing of the key.  Decoded rows and the first row of a
    portion, around page borders."""
    dim, rot_dim, heads = 16, 16, 3

    def plant(spans, qd, rows, s, rot):
        at = 0
        for b, (st, n) in enumerate(spans):
            p = st - window + (1 if inside else 0)
            D = s.dim + s.rot_dim
            x = qd[at, :heads * D].float().view(heads, D)
            x[:, s.dim:] = x[0, s.dim:]                                   # the heads share the rotated query part
            qd[at, :heads * D] = x.reshape(-1).to(dtype)
            qr = O.rotate_half(x[:1, None, s.dim:].reshape(1, 1, -1), torch.tensor([st]), rot).reshape(-1)
            rows[b][p, s.rank:] = (qr * 9.0).to(dtype)
            at += n

    for spans in ([(st, 1) for st in (window, 319, 320, 321, 383, 384)], [(window + 1, 1), (320, 2), (384, 130)]):
        got, want = attention_case(spans, heads, dim, rot_dim, 24, 40, window, dtype, sink=0.0, plant=plant, seed=window)
        at = 0
        for st, n in spans:
            assert rel(got[at], want[at]) < (2e-5 if dtype == torch.float32 else 1.5e-2), (st, n)
            at += n
        other, _ = attention_case(spans, heads, dim, rot_dim, 24, 40, window + (-1 if inside else 1), dtype, sink=0.0,
                                  plant=lambda *a: plant(*a), seed=window)
        assert rel(other[0], got[0]) > 0.2                                # (the planted key decides the row)


@pytest.mark.parametrize("sink", [-30.0, 0.0, 7.0])
def test_sink_mass(sink):
    """A sink above every score takes almost all of the weight; one far below changes nothing."""
    spans = [(100, 1), (30, 40)]
    got, want = attention_case(spans, 3, 16, 8, 24, 40, 50, torch.float32, sink=sink)
    assert rel(got, want) < 2e-5
    none, _ = attention_case(spans, 3, 16, 8, 24, 40, 50, torch.float32, sink=-1e4)
    assert (rel(got, none) < 1e-6) == (sink == -30.0)


def test_decode_key_splits():
    """Long contexts: the keys of one row are shared by several CTAs, the sink counts once."""
    for spans, window in (([(1500, 1), (700, 1)], 600), ([(1999, 1)], 0), ([(64 * i + 5, 1) for i in range(40)], 333)):
        got, want = attention_case(spans, 20, 32, 16, 32, 128, window, torch.bfloat16, sink=3.0)
        assert rel(got, want) < 1.2e-2


def test_expanded_heads_in_groups(monkeypatch):
    monkeypatch.setattr(L, "EXPAND_BUDGET_BYTES", 2 * 170 * (32 + 48) * 2)
    got, want = attention_case([(100, 70)], 5, 32, 16, 48, 64, 0, torch.bfloat16)
    assert rel(got, want) < 1.2e-2


# ---- whole models through the engine ----------------------------------------------------------------------------------

@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_engine_schedules(name, dtype):
    """Whole prompt, portions down to two tokens, token by token: all positions against the plain forward."""
    raw, low = CONFIGS[name]
    t = O.random_tensors(raw, 1, low)
    ids = random_ids(raw, 200, 2)
    want = O.forward(raw, t, ids)
    eng = make_engine(raw, t, "cuda", dtype)
    for cuts in ([200], portions(200, [2, 64, 3, 29, 70]), portions(200, [150], tail=40), [1] * 200):
        err = row_error(feed(eng, ids, cuts), want)
        # (heads of eight values: a norm over a few rounded numbers now and then makes one position's error large)
        top = 0.3 if name == "ones" else 2 * BF16_TOL
        assert err.max() < (FP32_TOL if dtype == torch.float32 else top), (cuts[:5], err.argmax(), err.max())
        assert err.mean() < (FP32_TOL if dtype == torch.float32 else BF16_TOL / 2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_engine_mixed_batches_and_reused_slots(dtype):
    raw, low = CONFIGS["tiled"]
    t = O.random_tensors(raw, 3, low)
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
        assert err.max() < (FP32_TOL if dtype == torch.float32 else 2 * BF16_TOL), (i, err.max())


def far_key_model():
    """Nearly undamped recurrences, and attention rows sharpened, so that tokens hundreds of positions back stay in the logits."""
    raw, low = CONFIGS["tiled"]
    t = O.random_tensors(raw, 4, low)
    t["l2.mix.a2.b"] += 8.0
    t["l1.mix.f.b"] += 6.0
    for n in ("l0.mix.q", "l3.mix.q"):
        t[n] = t[n] * 3
    return raw, t


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_long_decoding(dtype):
    """Hundreds of decoded tokens over page borders and through the windows, in a graph."""
    raw, t = far_key_model()
    ids = random_ids(raw, 420, 6)
    want = O.forward(raw, t, ids)
    changed = O.forward(raw, t, [(ids[0] + 1) % raw["vocab"]] + ids[1:])
    assert row_error(changed, want)[-1] > 0.02                            # the first token still matters at the end
    err = row_error(feed(make_engine(raw, t, "cuda", dtype), ids, [60] + [1] * 360), want)
    assert err.max() < (1e-4 if dtype == torch.float32 else 2.5 * BF16_TOL), (err.argmax(), err.max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_greedy_generation_through_the_scheduler(dtype):
    from slopllm_b200.config import SamplingParams
    from slopllm_b200.sampling.workspace import SamplingWorkspace
    from slopllm_b200.scheduler.scheduler import GenerationRequest, GenerationScheduler
    raw, low = CONFIGS["wide"]
    t = O.random_tensors(raw, 7, low)
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
        assert (best - took).max() <= (1e-4 if dtype == torch.float32 else 0.15) * logits.std(), r.id
    assert eng.model.states.free == 3


def test_trace_replay_program(tmp_path):
    """`bin/trace_run` as a user starts it."""
    import json
    import os
    import subprocess
    import numpy as np
    from test_gidisun import write_checkpoint
    raw, low = CONFIGS["wide"]
    t = O.random_tensors(raw, 2, low)
    model_dir = write_checkpoint(tmp_path / "m", raw, t)
    ids = random_ids(raw, 100, 1)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:98], "want": [5, 97]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": ids[98:99], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": ids[99:], "want": [0]}], "end": ["a"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    p = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", model_dir, "--dtype", "bfloat16", "--out", str(tmp_path), "--max-tokens", "128"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    got = torch.cat([torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4")).view(-1, raw["vocab"]) for i in (0, 2)])
    assert row_error(got, O.forward(raw, t, ids)[[5, 97, 99]]).max() < 2 * BF16_TOL
