"""Recurrent sub-layer ops of the hybrid families: Gated DeltaNet (Qwen3.5), KDA and manifold
hyper-connections (glm5_next), GLA and mLSTM (Gidisun), retention and minGRU (Vononex).  CUDA tensors run the sm_100a kernels of
`csrc/recurrent.cu`, `csrc/gated_scan.cu`, `csrc/gated_chunk.cu` and `csrc/min_gru.cu`;
CPU tensors run the fp32 definitions in `ops/reference.py` (the oracle of the GPU tests).
"""
from __future__ import annotations

import ctypes as C
import math
from typing import Optional

import torch

from . import reference as R
from .rotary import Turn


class GdnParams(C.Structure):
    _fields_ = [("out", C.c_void_p), ("state", C.c_void_p), ("qkv", C.c_void_p), ("ld_qkv", C.c_int), ("a", C.c_void_p),
                ("b", C.c_void_p), ("A_log", C.c_void_p), ("dt_bias", C.c_void_p), ("g", C.c_void_p), ("qo_indptr", C.c_void_p),
                ("state_idx", C.c_void_p), ("h", C.c_int), ("dk", C.c_int), ("dv", C.c_int), ("normalize_qk", C.c_int),
                ("lower_bound", C.c_float), ("norm_eps", C.c_float)]


def _native():
    from . import native as N
    return N


def _split_qkv(qkv, h, dk, dv):
    T = qkv.shape[0]
    q = qkv[:, :h * dk].reshape(T, h, dk)
    k = qkv[:, h * dk:2 * h * dk].reshape(T, h, dk)
    v = qkv[:, 2 * h * dk:2 * h * dk + h * dv].reshape(T, h, dv)
    return q, k, v


def gdn_scan(qkv, a, b, A_log, dt_bias, state, qo_indptr, state_idx, h: int, dk: int, dv: int):
    """Gated DeltaNet over the token ranges of B sequences (a decode step is one token each).

    qkv [T, h*dk | h*dk | h*dv] (conv output), a/b [T, h], A_log/dt_bias [h] fp32, state
    [slots, h, dk, dv] fp32 updated in place, qo_indptr [B+1], state_idx [B].  q is
    L2-normalised and scaled by dk^-0.5, k L2-normalised, beta = sigmoid(b),
    decay = exp(-exp(A_log) * softplus(a + dt_bias)).  Returns [T, h, dv] bf16.
    """
    T = qkv.shape[0]
    if qkv.is_cuda:
        N = _native()
        out = torch.empty(T, h, dv, dtype=torch.bfloat16, device=qkv.device)
        p = GdnParams(out=out.data_ptr(), state=state.data_ptr(), qkv=qkv.data_ptr(), ld_qkv=qkv.stride(0), a=a.data_ptr(),
                      b=b.data_ptr(), A_log=A_log.data_ptr(), dt_bias=dt_bias.data_ptr(), g=0, qo_indptr=qo_indptr.data_ptr(),
                      state_idx=state_idx.data_ptr(), h=h, dk=dk, dv=dv, normalize_qk=1, lower_bound=0.0, norm_eps=1e-8)
        N.call("sl_delta_scan", C.byref(p), qo_indptr.numel() - 1, N.stream())
        return out
    q, k, v = _split_qkv(qkv.to(torch.float32), h, dk, dv)
    q = q * torch.rsqrt((q * q).sum(-1, keepdim=True) + 1e-8) * dk ** -0.5
    k = k * torch.rsqrt((k * k).sum(-1, keepdim=True) + 1e-8)
    beta = torch.sigmoid(b.to(torch.float32))
    g = -torch.exp(A_log.to(torch.float32)) * torch.nn.functional.softplus(a.to(torch.float32) + dt_bias.to(torch.float32))
    out = torch.empty(T, h, dv, dtype=torch.float32, device=qkv.device)
    ind = qo_indptr.tolist()
    for bi in range(len(ind) - 1):
        lo, hi = ind[bi], ind[bi + 1]
        if hi > lo:
            slot = int(state_idx[bi])
            out[lo:hi], state[slot] = R.gdn_recurrent(q[lo:hi], k[lo:hi], v[lo:hi], g[lo:hi], beta[lo:hi], state[slot])
    return out.to(torch.bfloat16)


def kda_scan(qkv, forget, b, A_log, dt_bias, state, qo_indptr, state_idx, h: int, dk: int, dv: int, lower_bound: float):
    """KDA recurrence: as :func:`gdn_scan` but with a per-channel decay
    exp(lower_bound * sigmoid(exp(A_log[h]) * (forget[t, h, :] + dt_bias[h, :]))), lower_bound < 0.
    qkv [T, h*dk | h*dk | h*dv] (conv outputs), forget [T, h, dk] bf16, b [T, h], dt_bias [h, dk] fp32."""
    if not lower_bound < 0:
        raise ValueError("kda_scan: the gate lower bound must be negative and finite")
    T = qkv.shape[0]
    if qkv.is_cuda:
        N = _native()
        out = torch.empty(T, h, dv, dtype=torch.bfloat16, device=qkv.device)
        forget = forget.to(torch.bfloat16).contiguous()
        p = GdnParams(out=out.data_ptr(), state=state.data_ptr(), qkv=qkv.data_ptr(), ld_qkv=qkv.stride(0), a=0, b=b.data_ptr(),
                      A_log=A_log.data_ptr(), dt_bias=dt_bias.contiguous().data_ptr(), g=forget.data_ptr(),
                      qo_indptr=qo_indptr.data_ptr(), state_idx=state_idx.data_ptr(), h=h, dk=dk, dv=dv, normalize_qk=1,
                      lower_bound=float(lower_bound), norm_eps=1e-6)
        N.call("sl_delta_scan", C.byref(p), qo_indptr.numel() - 1, N.stream())
        return out
    q, k, v = _split_qkv(qkv.to(torch.float32), h, dk, dv)
    out = torch.empty(T, h, dv, dtype=torch.float32, device=qkv.device)
    ind = qo_indptr.tolist()
    for bi in range(len(ind) - 1):
        lo, hi = ind[bi], ind[bi + 1]
        if hi > lo:
            slot = int(state_idx[bi])
            out[lo:hi], state[slot] = R.kda_scan(q[lo:hi], k[lo:hi], v[lo:hi], forget[lo:hi].reshape(hi - lo, h, dk), b[lo:hi], A_log,
                                                 dt_bias.reshape(h, dk), state[slot], lower_bound)
    return out.to(torch.bfloat16)


# ---- gated outer-product recurrences: GLA, mLSTM, retention --------------------------------------------------------------------------

class GatedScanParams(C.Structure):
    _fields_ = [("out", C.c_void_p), ("q", C.c_void_p), ("k", C.c_void_p), ("v", C.c_void_p), ("g", C.c_void_p), ("ld", C.c_int),
                ("gates", C.c_void_p), ("ld_gates", C.c_int), ("a2", C.c_void_p), ("a2_b", C.c_void_p), ("rank", C.c_int),
                ("inv_tau", C.c_float), ("i_b", C.c_void_p), ("f_b", C.c_void_p), ("cap", C.c_float), ("norm_w", C.c_void_p),
                ("eps", C.c_float), ("S", C.c_void_p), ("n", C.c_void_p), ("m", C.c_void_p), ("qo_indptr", C.c_void_p),
                ("state_idx", C.c_void_p), ("h", C.c_int), ("dk", C.c_int), ("dv", C.c_int), ("ldg", C.c_int), ("ldo", C.c_int),
                ("group", C.c_int), ("decay", C.c_void_p), ("turn", C.c_void_p), ("ldt", C.c_int), ("rot_dims", C.c_int),
                ("out_scale", C.c_float)]


KIND_GLA, KIND_MLSTM, KIND_RETENTION = 0, 1, 2
CHUNK = 64                          # tokens per chunk of the chunked kernels
CHUNK_MIN_Q = 16                    # longest portion of a step from which on they are used
CHUNK_SCRATCH_BYTES = 96 << 20      # chunk states of one pass (they stay in L2); longer steps run in several passes


class GatedChunkParams(C.Structure):
    _fields_ = [("s", GatedScanParams), ("chunks", C.c_void_p), ("seq_chunks", C.c_void_p), ("c0", C.c_int), ("c1", C.c_int),
                ("b", C.c_void_p), ("loc", C.c_void_p), ("nloc", C.c_void_p), ("scal", C.c_void_p), ("slab", C.c_int), ("slab_bufs", C.c_int)]


class ChunkPlan:
    """The chunks of a step's portions: table [chunks, 4] of (sequence, first token, tokens, last chunk of its sequence) and
    the chunk range of every sequence, on the device."""

    def __init__(self, lengths, device):
        rows, ends, t0 = [], [0], 0
        for b, n in enumerate(lengths):
            for o in range(0, n, CHUNK):
                rows.append((b, t0 + o, min(CHUNK, n - o), int(o + CHUNK >= n)))
            ends.append(len(rows))
            t0 += n
        self.count, self.longest = len(rows), max(lengths)
        flat = [x for r in rows for x in r] + ends
        t = torch.tensor(flat, dtype=torch.int32, device=device)
        self.table, self.seq_chunks = t[:4 * self.count], t[4 * self.count:]

    @staticmethod
    def of(st):
        """The plan of a step that holds portions of prompts (made once per step), else None."""
        spans = st.extra.get("spans")
        if spans is None or not st.input_ids.is_cuda:
            return None
        if "chunk_plan" not in st.extra:
            st.extra["chunk_plan"] = ChunkPlan([n for _, n in spans], st.input_ids.device)
        return st.extra["chunk_plan"]


def _gated_params(p_in, h, dk, dv, out, norm_w, eps, qo_indptr, state_idx) -> GatedScanParams:
    esz = p_in.element_size()
    base = p_in.data_ptr()
    return GatedScanParams(out=out.data_ptr(), ldo=out.stride(0), q=base, k=base + h * dk * esz, v=base + 2 * h * dk * esz,
                           g=base + (2 * h * dk + h * dv) * esz, ld=p_in.stride(0), norm_w=_native().ptr(norm_w), eps=float(eps),
                           qo_indptr=qo_indptr.data_ptr(), state_idx=state_idx.data_ptr(), h=h, dk=dk, dv=dv)


def _run_gated(kind: int, p: GatedScanParams, proj, out, qo_indptr, plan=None) -> torch.Tensor:
    N = _native()
    B = qo_indptr.numel() - 1
    h, dk, dv, dev = p.h, p.dk, p.dv, proj.device
    if (plan is None or plan.longest < CHUNK_MIN_Q or proj.dtype != torch.bfloat16 or out.dtype != torch.bfloat16 or p.ld % 8
            or p.q % 16 or p.ldo % 2 or p.out % 4 or not N.fn("sl_gated_chunk_ok")(kind, dk, dv, p.rank)):
        N.call("sl_gated_step", C.byref(p), B, kind, int(proj.dtype == torch.float32), int(out.dtype == torch.float32), N.stream())
        return out
    per_pass = min(plan.count, max(1, CHUNK_SCRATCH_BYTES // (h * dk * dv * 4)))
    loc = torch.empty(per_pass * h * dk * dv, dtype=torch.float32, device=dev)
    b = torch.empty(out.shape[0] * h * dk if kind == KIND_GLA else 1, dtype=torch.float32, device=dev)
    aux = torch.empty(per_pass * h * (dk + 4) if kind == KIND_MLSTM else 1, dtype=torch.float32, device=dev)
    cp = GatedChunkParams(s=p, chunks=plan.table.data_ptr(), seq_chunks=plan.seq_chunks.data_ptr(), b=b.data_ptr(), loc=loc.data_ptr(),
                          nloc=aux.data_ptr(), scal=aux.data_ptr() + per_pass * h * dk * 4)
    for c0 in range(0, plan.count, per_pass):
        cp.c0, cp.c1 = c0, min(plan.count, c0 + per_pass)
        N.call("sl_gated_chunks", C.byref(cp), B, kind, N.stream())
    return out


def _qkvg(proj, h, dk, dv):
    T = proj.shape[0]
    q, k, v, g = torch.split(proj[:, :h * (2 * dk + 2 * dv)].to(torch.float32), [h * dk, h * dk, h * dv, h * dv], dim=1)
    return q.reshape(T, h, dk) * dk ** -0.5, k.reshape(T, h, dk), v.reshape(T, h, dv), g.reshape(T, h, dv)


def gla_mix(proj, low, a2, a2_b, tau: float, norm_w, eps: float, state, qo_indptr, state_idx, h: int, dk: int, dv: int, out_dtype,
            plan=None):
    """Gated linear attention over the token ranges of B sequences, up to the output projection.

    proj [T, h*dk (q) | h*dk (k) | h*dv (v) | h*dv (output gate)], low fp32 [T, rank] the low-rank decay input, a2 [h*dk, rank],
    a2_b fp32 [h*dk], norm_w fp32 [dv] shared by the heads, state [slots, h, dk, dv] fp32 updated in place.
    S = diag(sigmoid(a2 low + b)^(1/tau)) S + k v^T, o = S^T q dk^-0.5; returns rms(o) * norm_w * silu(gate) [T, h*dv].
    With a :class:`ChunkPlan` longer portions run in chunks on the tensor cores (`csrc/gated_chunk.cu`)."""
    T = proj.shape[0]
    if proj.is_cuda:
        out = torch.empty(T, h * dv, dtype=out_dtype, device=proj.device)
        p = _gated_params(proj, h, dk, dv, out, norm_w, eps, qo_indptr, state_idx)
        p.gates, p.ld_gates, p.a2, p.a2_b, p.rank, p.inv_tau = low.data_ptr(), low.stride(0), a2.data_ptr(), a2_b.data_ptr(), a2.shape[1], 1.0 / tau
        p.S = state.data_ptr()
        return _run_gated(KIND_GLA, p, proj, out, qo_indptr, plan)
    q, k, v, g = _qkvg(proj, h, dk, dv)
    z = low.to(torch.float32) @ a2.to(torch.float32).t() + a2_b
    decay = torch.exp(torch.nn.functional.logsigmoid(z) / tau).view(T, h, dk)
    o = torch.empty(T, h, dv, dtype=torch.float32)
    ind = qo_indptr.tolist()
    for b in range(len(ind) - 1):
        if ind[b + 1] > ind[b]:
            o[ind[b]:ind[b + 1]] = R.gla_scan(q[ind[b]:ind[b + 1]], k[ind[b]:ind[b + 1]], v[ind[b]:ind[b + 1]], decay[ind[b]:ind[b + 1]],
                                              state[int(state_idx[b])])
    o = R.rmsnorm(o, norm_w, eps) * torch.nn.functional.silu(g)
    return o.reshape(T, h * dv).to(out_dtype)


def mlstm_mix(proj, gates, i_b, f_b, cap: float, norm_w, eps: float, state, qo_indptr, state_idx, h: int, dk: int, dv: int, out_dtype,
            plan=None):
    """mLSTM matrix memory over the token ranges of B sequences, up to the output projection.

    proj as in :func:`gla_mix`, gates fp32 [T, i_raw h | f_raw h], i_b / f_b fp32 [h], norm_w fp32 [h*dv], state = (S
    [slots, h, dk, dv], n [slots, h, dk], m [slots, h]) fp32 updated in place.  Both gates pass a soft cap cap*tanh(x/cap), the
    forget gate then a log-sigmoid; the running maximum m keeps the exponentials below one.  Returns
    rms(o) * norm_w * sigmoid(gate) [T, h*dv]."""
    T = proj.shape[0]
    S, n, m = state
    if proj.is_cuda:
        out = torch.empty(T, h * dv, dtype=out_dtype, device=proj.device)
        p = _gated_params(proj, h, dk, dv, out, norm_w, eps, qo_indptr, state_idx)
        p.gates, p.ld_gates, p.i_b, p.f_b, p.cap = gates.data_ptr(), gates.stride(0), i_b.data_ptr(), f_b.data_ptr(), float(cap)
        p.S, p.n, p.m = S.data_ptr(), n.data_ptr(), m.data_ptr()
        return _run_gated(KIND_MLSTM, p, proj, out, qo_indptr, plan)
    q, k, v, g = _qkvg(proj, h, dk, dv)
    gi = cap * torch.tanh((gates[:, :h].to(torch.float32) + i_b) / cap)
    gf = torch.nn.functional.logsigmoid(cap * torch.tanh((gates[:, h:2 * h].to(torch.float32) + f_b) / cap))
    o = torch.empty(T, h, dv, dtype=torch.float32)
    ind = qo_indptr.tolist()
    for b in range(len(ind) - 1):
        r, sl = slice(ind[b], ind[b + 1]), int(state_idx[b])
        if ind[b + 1] > ind[b]:
            o[r] = R.mlstm_scan(q[r], k[r], v[r], gi[r], gf[r], S[sl], n[sl], m[sl])
    o = R.rmsnorm(o, torch.ones(dv), eps).reshape(T, h * dv) * norm_w * torch.sigmoid(g.reshape(T, h * dv))
    return o.to(out_dtype)


def retention_decays(decay) -> torch.Tensor:
    """[2, heads] fp32 for :func:`retention_mix`: each head's decay and its log2, made once on the host (2^-200 stands for nothing kept)."""
    if any(not 0.0 <= d for d in decay):
        raise ValueError("decays must not be negative")
    return torch.tensor([list(decay), [math.log2(d) if d > 0 else -200.0 for d in decay]], dtype=torch.float32)


def retention_mix(proj, decay, turn: Turn, angles, eps: float, state, qo_indptr, state_idx, h: int, dk: int, dv: int, out, scale: float = 1.0,
                  plan=None) -> None:
    """Retention over the token ranges of B sequences, up to the output projection: linear attention with a fixed decay per head.

    proj [T, h*dk (q) | h*dk (k) | h*dv (v) | h*dv (output gate)], q and k rows in the adjacent order of `ops/rotary.py` and turned by
    `turn`; decay from :func:`retention_decays`; state [slots, h, dk, dv] fp32 updated in place.
    S = decay S + k v^T, o = S^T q dk^-0.5; out [T, h*dv] (rows of any stride) = scale * rms(o) * silu(gate)."""
    T = proj.shape[0]
    if proj.is_cuda:
        p = _gated_params(proj, h, dk, dv, out, None, eps, qo_indptr, state_idx)
        p.S, p.decay, p.turn, p.ldt, p.rot_dims = state.data_ptr(), decay.data_ptr(), angles.data_ptr() + turn.at * 8, angles.shape[1], turn.dims
        p.out_scale = scale
        _run_gated(KIND_RETENTION, p, proj, out, qo_indptr, plan)
        return
    q, k, v, g = _qkvg(proj, h, dk, dv)
    q, k = turn.apply(q, angles), turn.apply(k, angles)
    keep = decay[0].view(1, h, 1).expand(T, h, dk)
    o = torch.empty(T, h, dv, dtype=torch.float32)
    ind = qo_indptr.tolist()
    for b in range(len(ind) - 1):
        r = slice(ind[b], ind[b + 1])
        if ind[b + 1] > ind[b]:
            o[r] = R.gla_scan(q[r], k[r], v[r], keep[r], state[int(state_idx[b])])
    o = R.rmsnorm(o, torch.ones(dv), eps) * torch.nn.functional.silu(g) * scale
    out.copy_(o.reshape(T, h * dv))


# ---- element-wise gated recurrence: minGRU -----------------------------------------------------------------------------------

class MinGruParams(C.Structure):
    _fields_ = [("out", C.c_void_p), ("ldo", C.c_int), ("z", C.c_void_p), ("u", C.c_void_p), ("g", C.c_void_p), ("ld", C.c_int),
                ("z_b", C.c_void_p), ("u_b", C.c_void_p), ("S", C.c_void_p), ("qo_indptr", C.c_void_p), ("state_idx", C.c_void_p),
                ("W", C.c_int), ("chunks", C.c_void_p), ("seq_chunks", C.c_void_p), ("maps", C.c_void_p), ("start", C.c_void_p)]


def min_gru_mix(proj, bias: Optional[torch.Tensor], state, qo_indptr, state_idx, W: int, out_dtype, plan=None) -> torch.Tensor:
    """minGRU over the token ranges of B sequences, up to the output projection.

    proj [T, W (z) | W (u) | W (output gate)], bias fp32 [W (z) | W (u)], state [slots, W] fp32 updated in place.
    z = sigmoid(z), c = u + 1/2 where u >= 0 and sigmoid(u) elsewhere, S = (1 - z) S + z c; returns S * silu(gate) [T, W].
    With a :class:`ChunkPlan` longer portions run in chunks that are composed."""
    T = proj.shape[0]
    if proj.is_cuda:
        N = _native()
        out = torch.empty(T, W, dtype=out_dtype, device=proj.device)
        at = lambda i: proj.data_ptr() + i * W * proj.element_size()
        p = MinGruParams(out=out.data_ptr(), ldo=out.stride(0), z=at(0), u=at(1), g=at(2), ld=proj.stride(0), z_b=N.ptr(bias),
                         u_b=0 if bias is None else bias.data_ptr() + 4 * W, S=state.data_ptr(), qo_indptr=qo_indptr.data_ptr(),
                         state_idx=state_idx.data_ptr(), W=W)
        B, types = qo_indptr.numel() - 1, (int(proj.dtype == torch.float32), int(out_dtype == torch.float32))
        if plan is None or plan.longest < CHUNK_MIN_Q:
            N.call("sl_min_gru_step", C.byref(p), B, *types, N.stream())
            return out
        scratch = torch.empty(plan.count * W * 2 + B * W, dtype=torch.float32, device=proj.device)
        p.chunks, p.seq_chunks = plan.table.data_ptr(), plan.seq_chunks.data_ptr()
        p.maps, p.start = scratch.data_ptr(), scratch.data_ptr() + plan.count * W * 8
        N.call("sl_min_gru_chunks", C.byref(p), plan.count, *types, N.stream())
        return out
    x = proj[:, :3 * W].to(torch.float32)
    z, u, g = x[:, :W], x[:, W:2 * W], x[:, 2 * W:]
    if bias is not None:
        z, u = z + bias[:W], u + bias[W:]
    S = torch.empty(T, W, dtype=torch.float32)
    ind = qo_indptr.tolist()
    for b in range(len(ind) - 1):
        r = slice(ind[b], ind[b + 1])
        if ind[b + 1] > ind[b]:
            S[r] = R.min_gru_scan(z[r], u[r], state[int(state_idx[b])])
    return (S * torch.nn.functional.silu(g)).to(out_dtype)


def causal_conv1d(x, weight, bias, state, qo_indptr, state_idx, activation: bool = True):
    """Depthwise causal conv over each sequence's tokens with rolling state [slots, C, Kw-1]
    (fp32, updated in place).  x [T, C] -> [T, C] bf16."""
    T, Cc = x.shape
    Kw = weight.shape[1]
    if x.is_cuda:
        N = _native()
        y = torch.empty(T, Cc, dtype=torch.bfloat16, device=x.device)
        N.call("sl_causal_conv1d", y.data_ptr(), state.data_ptr(), x.data_ptr(), weight.data_ptr(), N.ptr(bias),
               qo_indptr.data_ptr(), state_idx.data_ptr(), qo_indptr.numel() - 1, Cc, Kw, x.stride(0), int(activation), N.stream())
        return y
    y = torch.empty(T, Cc, dtype=torch.float32, device=x.device)
    ind = qo_indptr.tolist()
    for bi in range(len(ind) - 1):
        lo, hi = ind[bi], ind[bi + 1]
        if hi > lo:
            slot = int(state_idx[bi])
            y[lo:hi], state[slot] = R.causal_conv1d(x[lo:hi], weight, bias, state[slot], activation)
    return y.to(torch.bfloat16)


def rmsnorm_gated(x, gate, weight, eps: float, sigmoid_gate: bool = False):
    """rmsnorm(x) * w * silu(gate)  (sigmoid(gate) for KDA) over the last dim; x, gate [rows, D]."""
    if x.is_cuda:
        N = _native()
        x, gate = x.contiguous(), gate.contiguous()
        out = torch.empty_like(x)
        N.call("sl_rmsnorm_gated", out.data_ptr(), x.data_ptr(), gate.data_ptr(), weight.data_ptr(), x.shape[0], x.shape[1],
               float(eps), int(sigmoid_gate), N.stream())
        return out
    f = R.kda_norm if sigmoid_gate else R.rmsnorm_gated
    return f(x, gate, weight, eps).to(x.dtype)


def mhc_pre(x, fn, base, scale, norm_eps: float, hc_eps: float, iters: int):
    """x [T, 4, H] bf16 residual streams -> (collapsed [T, H] bf16, post [T, 4] f32, comb [T, 4, 4] f32)."""
    if x.dim() != 3 or x.shape[1] != 4 or not norm_eps > 0 or not hc_eps > 0 or iters < 1:
        raise ValueError("mhc_pre: expected [tokens, 4, hidden] and positive epsilons / iteration count")
    T, _, H = x.shape
    if tuple(fn.shape) != (24, 4 * H) or base.numel() != 24 or scale.numel() != 3:
        raise ValueError("mhc_pre: expected fn [24, 4*hidden], base [24], scale [3]")
    if x.is_cuda:
        N = _native()
        collapsed = torch.empty(T, H, dtype=torch.bfloat16, device=x.device)
        post = torch.empty(T, 4, dtype=torch.float32, device=x.device)
        comb = torch.empty(T, 4, 4, dtype=torch.float32, device=x.device)
        N.call("sl_mhc_pre", collapsed.data_ptr(), post.data_ptr(), comb.data_ptr(), x.to(torch.bfloat16).contiguous().data_ptr(),
               fn.to(torch.bfloat16).contiguous().data_ptr(), base.to(torch.float32).contiguous().data_ptr(),
               scale.to(torch.float32).contiguous().data_ptr(), T, H, float(norm_eps), float(hc_eps), int(iters), N.stream())
        return collapsed, post, comb
    collapsed, post, comb = R.mhc_pre(x, fn, base, scale, norm_eps, hc_eps, iters)
    return collapsed.to(torch.bfloat16), post, comb


def mhc_post(residual, block, post, comb):
    """residual [T, 4, H], block [T, H] -> new streams [T, 4, H] bf16."""
    if residual.dim() != 3 or residual.shape[1] != 4:
        raise ValueError("mhc_post: expected [tokens, 4, hidden]")
    if residual.is_cuda:
        N = _native()
        T, _, H = residual.shape
        out = torch.empty(T, 4, H, dtype=torch.bfloat16, device=residual.device)
        N.call("sl_mhc_post", out.data_ptr(), residual.to(torch.bfloat16).contiguous().data_ptr(),
               block.to(torch.bfloat16).contiguous().data_ptr(), post.contiguous().data_ptr(), comb.contiguous().data_ptr(), T, H,
               N.stream())
        return out
    return R.mhc_post(residual, block, post, comb).to(torch.bfloat16)


def mhc_streams(x, expand: bool):
    """expand: [T, H] -> [T, 4, H] (copies); collapse: [T, 4, H] -> [T, H] (mean)."""
    if (x.dim() != 2) if expand else (x.dim() != 3 or x.shape[1] != 4):
        raise ValueError("mhc_streams: expected [tokens, hidden] to expand or [tokens, 4, hidden] to collapse")
    if x.is_cuda:
        N = _native()
        T, H = x.shape[0], x.shape[-1]
        out = torch.empty((T, 4, H) if expand else (T, H), dtype=torch.bfloat16, device=x.device)
        N.call("sl_mhc_streams", out.data_ptr(), x.to(torch.bfloat16).contiguous().data_ptr(), T, H, int(expand), N.stream())
        return out
    return R.mhc_streams(x, expand).to(torch.bfloat16)
