"""Gated delta rule with one decay per key channel (and its short convolutions), up to the output projection.

    S = diag(g_t) S;  u = beta_t (v_t - S^T k_t);  S = S + k_t u^T;  o_t = S^T q_t

q, k, v pass a causal convolution over the last `taps` inputs of their channel and silu, q and k become unit vectors per head
(q also times dk^-0.5), g = exp(-exp(A_log) softplus(a2 low_a + dt_bias)), beta = sigmoid(b).  The result is
rms(o) * norm * sigmoid(g2 low_g).  Query / key heads may be shared by several value heads.

Per sequence: the fp32 state S and the last inputs of the convolutions in a ring, input of position p in row p % taps.

CUDA tensors run `csrc/short_conv.cu`, `csrc/delta_step.cu` (token by token: decoding, fp32, any sizes) and
`csrc/delta_chunk.cu` (chunks of 64 tokens on the tensor cores); CPU tensors run the fp32 definition below.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch

UNIT_EPS = 1e-6


def _native():
    from . import native as N
    return N


class DeltaStepParams(C.Structure):
    _fields_ = [("out", C.c_void_p), ("ldo", C.c_int), ("q", C.c_void_p), ("k", C.c_void_p), ("v", C.c_void_p), ("ld", C.c_int),
                ("low", C.c_void_p), ("ld_low", C.c_int), ("ra", C.c_int), ("rg", C.c_int), ("b", C.c_void_p), ("a2", C.c_void_p),
                ("g2", C.c_void_p), ("dt_bias", C.c_void_p), ("A_log", C.c_void_p), ("norm_w", C.c_void_p), ("eps", C.c_float),
                ("unit_eps", C.c_float), ("S", C.c_void_p), ("conv_w", C.c_void_p), ("conv", C.c_void_p), ("taps", C.c_int),
                ("positions", C.c_void_p), ("qo_indptr", C.c_void_p), ("state_idx", C.c_void_p), ("h", C.c_int), ("hk", C.c_int),
                ("dk", C.c_int), ("dv", C.c_int)]


@dataclass
class DeltaShape:
    heads: int                 # value heads of this rank
    kv_heads: int              # query / key heads of this rank
    dk: int
    dv: int
    taps: int
    eps: float

    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dk + self.heads * self.dv


@dataclass
class DeltaWeights:
    conv: torch.Tensor         # fp32 [taps, channels] (q | k | v), last row: the current token
    a2: torch.Tensor           # [heads * dk, rank of the decay]
    g2: torch.Tensor           # [heads * dv, rank of the gate]
    dt_bias: torch.Tensor      # fp32 [heads * dk]
    A_log: torch.Tensor        # fp32 [heads]
    norm: torch.Tensor         # fp32 [dv]


def short_conv(x: torch.Tensor, w: torch.Tensor, state: torch.Tensor, positions, qo_indptr, state_idx, longest: int, dtype) -> torch.Tensor:
    """silu of the causal convolution of every channel over the token ranges of B sequences; x [T, C] (rows of any stride), w fp32
    [taps, C], state fp32 [slots, taps, C] advanced in place.  Returns [T, C] in `dtype`."""
    T, Cn = x.shape
    taps = w.shape[0]
    if x.is_cuda:
        N = _native()
        y = torch.empty(T, Cn, dtype=dtype, device=x.device)
        N.call("sl_short_conv", y.data_ptr(), x.data_ptr(), x.stride(0), w.data_ptr(), state.data_ptr(), positions.data_ptr(), qo_indptr.data_ptr(),
               state_idx.data_ptr(), qo_indptr.numel() - 1, int(longest), Cn, taps, int(x.dtype == torch.float32), int(dtype == torch.float32),
               N.stream())
        return y
    y = torch.empty(T, Cn, dtype=torch.float32)
    ind = qo_indptr.tolist()
    for b in range(len(ind) - 1):
        lo, hi, ring = ind[b], ind[b + 1], state[int(state_idx[b])]
        if hi == lo:
            continue
        start = int(positions[lo])
        back = [ring[(start - j) % taps] for j in range(taps - 1, 0, -1)]          # (a slot not yet written holds zeros)
        full = torch.stack(back + list(x[lo:hi].to(torch.float32)))
        y[lo:hi] = sum(full[j:j + hi - lo] * w[j] for j in range(taps))
        for i in range(max(0, hi - lo - taps), hi - lo):
            ring[(start + i) % taps] = x[lo + i].to(torch.float32)
    return torch.nn.functional.silu(y).to(dtype)


def _low_rank(fine, ra, rg, h):
    return fine[:, :ra], fine[:, ra:ra + rg], fine[:, ra + rg:ra + rg + h]


def channel_delta_mix(main: torch.Tensor, fine: torch.Tensor, s: DeltaShape, w: DeltaWeights, S: torch.Tensor, conv: torch.Tensor, st,
                      qo_indptr, state_idx, out: torch.Tensor, ops, plan=None) -> None:
    """main [T, q | k | v channels], fine fp32 [T, decay rank | gate rank | heads (beta)]; result into `out` [T, heads * dv] (rows
    of any stride).  With a :class:`~slopllm_b200.ops.recurrent.ChunkPlan` longer portions run in chunks."""
    T, h, dk, dv = main.shape[0], s.heads, s.dk, s.dv
    ra, rg, qk = w.a2.shape[1], w.g2.shape[1], s.kv_heads * s.dk
    if main.is_cuda:
        from . import delta_chunk as DC
        portions = "spans" in st.extra
        longest = st.extra.get("max_q", 1)
        x = short_conv(main, w.conv, conv, st.positions, qo_indptr, state_idx, longest, out.dtype) if portions else main
        if portions and DC.usable(s, plan, x, out):
            DC.run(x, fine, s, w, S, qo_indptr, state_idx, out, ops, plan)
            return
        _step(x, fine, s, w, S, None if portions else conv, st, qo_indptr, state_idx, out)
        return
    x = short_conv(main, w.conv, conv, st.positions, qo_indptr, state_idx, 0, torch.float32)
    unit = lambda y: y / torch.sqrt((y * y).sum(-1, keepdim=True) + UNIT_EPS)
    grow = lambda y: unit(y.reshape(T, s.kv_heads, dk)).repeat_interleave(h // s.kv_heads, 1)
    q, k, v = grow(x[:, :qk]) * dk ** -0.5, grow(x[:, qk:2 * qk]), x[:, 2 * qk:].reshape(T, h, dv)
    la, lg, b = (y.to(torch.float32) for y in _low_rank(fine, ra, rg, h))
    z = la @ w.a2.to(torch.float32).t() + w.dt_bias
    decay = torch.exp(-torch.exp(w.A_log)[:, None] * torch.nn.functional.softplus(z).view(T, h, dk))
    beta, gate = torch.sigmoid(b), torch.sigmoid(lg @ w.g2.to(torch.float32).t())
    ind = qo_indptr.tolist()
    for i in range(len(ind) - 1):
        state = S[int(state_idx[i])]
        for t in range(ind[i], ind[i + 1]):
            state.mul_(decay[t].unsqueeze(-1))
            u = beta[t].unsqueeze(-1) * (v[t] - torch.einsum("hkv,hk->hv", state, k[t]))
            state.add_(k[t].unsqueeze(-1) * u.unsqueeze(-2))
            o = torch.einsum("hkv,hk->hv", state, q[t])
            o = o / torch.sqrt((o * o).mean(-1, keepdim=True) + s.eps) * w.norm
            out[t] = (o.reshape(-1) * gate[t]).to(out.dtype)


def _step(x, fine, s: DeltaShape, w: DeltaWeights, S, conv: Optional[torch.Tensor], st, qo_indptr, state_idx, out) -> None:
    """Token by token.  With `conv` (decoding: one token a sequence) the convolutions are part of the kernel and x holds the
    projections; otherwise x holds convolved rows."""
    N = _native()
    h, dk = s.heads, s.dk
    ra, rg, qk = w.a2.shape[1], w.g2.shape[1], s.kv_heads * dk
    at = lambda i: x.data_ptr() + i * x.element_size()
    p = DeltaStepParams(out=out.data_ptr(), ldo=out.stride(0), q=at(0), k=at(qk), v=at(2 * qk), ld=x.stride(0), low=fine.data_ptr(),
                        ld_low=fine.stride(0), ra=ra, rg=rg, b=fine.data_ptr() + 4 * (ra + rg), a2=w.a2.data_ptr(), g2=w.g2.data_ptr(),
                        dt_bias=w.dt_bias.data_ptr(), A_log=w.A_log.data_ptr(), norm_w=w.norm.data_ptr(), eps=s.eps, unit_eps=UNIT_EPS,
                        S=S.data_ptr(), conv_w=N.ptr(w.conv if conv is not None else None), conv=N.ptr(conv), taps=s.taps,
                        positions=st.positions.data_ptr(), qo_indptr=qo_indptr.data_ptr(), state_idx=state_idx.data_ptr(), h=h,
                        hk=s.kv_heads, dk=dk, dv=s.dv)
    N.call("sl_delta_step", C.byref(p), qo_indptr.numel() - 1, int(x.dtype == torch.float32), int(out.dtype == torch.float32), N.stream())
