"""Grouped-query attention over a paged cache with the options of recent small decoders: norm of queries and keys, any rotary
table, sliding window with kept first tokens, softmax sink, values of their own or the key projections themselves, values that
turn with their position.

A position sees the last `window` positions up to itself (0: all of them) and, whatever the distance, the first `keep_first`
ones.  CUDA tensors run `csrc/grouped_attn.cu` (and, for portions of prompts, the attention kernel of `csrc/latent_mma.cu` over
rows copied out of the pages); CPU tensors run the fp32 definition below.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch

from .dense import _slots
from .latent import PortionPlan, gather_rows, portion_attention
from .rotary import RotaryTable, Turn


def _native():
    from . import native as N
    return N


class GroupedPreParams(C.Structure):
    _fields_ = [("q", C.c_void_p), ("k", C.c_void_p), ("v", C.c_void_p), ("ld", C.c_int), ("heads", C.c_int), ("kv_heads", C.c_int),
                ("dim", C.c_int), ("vdim", C.c_int), ("rot_dims", C.c_int), ("q_norm", C.c_void_p), ("k_norm", C.c_void_p),
                ("freq", C.c_void_p), ("rot_gain", C.c_float), ("eps", C.c_float), ("positions", C.c_void_p), ("batch_idx", C.c_void_p),
                ("page_table", C.c_void_p), ("pt_stride", C.c_int), ("page_size", C.c_int), ("k_cache", C.c_void_p), ("v_cache", C.c_void_p),
                ("num_slots", C.c_int), ("q_out", C.c_void_p), ("guard", C.c_void_p), ("v_heads", C.c_int), ("q_bias", C.c_void_p),
                ("k_bias", C.c_void_p), ("v_bias", C.c_void_p)]


class GroupedAttnParams(C.Structure):
    _fields_ = [("q", C.c_void_p), ("k_cache", C.c_void_p), ("v_cache", C.c_void_p), ("num_slots", C.c_int), ("positions", C.c_void_p),
                ("batch_idx", C.c_void_p), ("page_table", C.c_void_p), ("pt_stride", C.c_int), ("page_size", C.c_int), ("heads", C.c_int),
                ("kv_heads", C.c_int), ("dim", C.c_int), ("vdim", C.c_int), ("window", C.c_int), ("keep_first", C.c_int),
                ("splits", C.c_int), ("scale", C.c_float), ("sink", C.c_void_p), ("out", C.c_void_p), ("ldo", C.c_int),
                ("o_part", C.c_void_p), ("lse_part", C.c_void_p), ("guard", C.c_void_p), ("turn", C.c_void_p), ("ldt", C.c_int),
                ("out_scale", C.c_float)]


class GroupedRowPreParams(C.Structure):
    _fields_ = [("q", C.c_void_p), ("k", C.c_void_p), ("v", C.c_void_p), ("ld", C.c_int), ("heads", C.c_int), ("kv_heads", C.c_int),
                ("dim", C.c_int), ("vdim", C.c_int), ("rot_dims", C.c_int), ("q_bias", C.c_void_p), ("k_bias", C.c_void_p),
                ("v_bias", C.c_void_p), ("q_norm", C.c_void_p), ("k_norm", C.c_void_p), ("sums", C.c_void_p), ("q_count", C.c_float),
                ("k_count", C.c_float), ("eps", C.c_float), ("gain", C.c_void_p), ("qk_turn", C.c_void_p), ("v_turn", C.c_void_p),
                ("ldt", C.c_int), ("positions", C.c_void_p), ("batch_idx", C.c_void_p), ("page_table", C.c_void_p), ("pt_stride", C.c_int),
                ("page_size", C.c_int), ("k_cache", C.c_void_p), ("v_cache", C.c_void_p), ("num_slots", C.c_int), ("q_out", C.c_void_p),
                ("guard", C.c_void_p)]


@dataclass
class GroupedShape:
    heads: int                 # query heads of this rank
    kv_heads: int              # key / value heads of this rank
    dim: int
    vdim: int
    scale: float
    window: int = 0
    keep_first: int = 0
    eps: float = 1e-5
    own_values: bool = True    # False: a value row is the key projection before norm and rotation (vdim == dim)
    v_heads: Optional[int] = None      # value heads of this rank, where they are not as many as its key heads


@dataclass
class GroupedWeights:
    q_norm: Optional[torch.Tensor]          # fp32 [dim], shared by the heads (None: no norm)
    k_norm: Optional[torch.Tensor]
    sink: Optional[torch.Tensor] = None     # fp32 [heads]
    bias: Optional[torch.Tensor] = None     # fp32, added to the projection rows


def _rms(x, w, eps):
    return x if w is None else x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def grouped_pre(proj: torch.Tensor, s: GroupedShape, w: GroupedWeights, rot: Optional[RotaryTable], st, k_cache: torch.Tensor,
                v_cache: torch.Tensor, dtype: torch.dtype) -> torch.Tensor:
    """proj [T, heads * dim (q) | kv_heads * dim (k) | kv_heads * vdim (v, if values are their own)] (`dtype` or fp32): norms and
    rotates queries and keys (`rot` None: does not), writes keys and values into their slots; returns the queries [T, heads, dim] in
    `dtype`.  Without key heads there are queries only."""
    T, kb = proj.shape[0], s.heads * s.dim
    vb = kb + s.kv_heads * s.dim
    nv = s.kv_heads if s.v_heads is None else s.v_heads
    if proj.is_cuda:
        N = _native()
        from . import tcgen05
        q = torch.empty(T, s.heads, s.dim, dtype=dtype, device=proj.device)
        at = lambda i: proj.data_ptr() + i * proj.element_size()
        bias = lambda i: 0 if w.bias is None else w.bias.data_ptr() + 4 * i
        v_at = vb if s.own_values else kb
        p = GroupedPreParams(q=at(0), k=at(kb), v=at(v_at), v_heads=nv, q_bias=bias(0), k_bias=bias(kb), v_bias=bias(v_at), ld=proj.stride(0), heads=s.heads, kv_heads=s.kv_heads,
                             dim=s.dim, vdim=s.vdim, rot_dims=0 if rot is None else rot.dims, q_norm=N.ptr(w.q_norm), k_norm=N.ptr(w.k_norm),
                             freq=0 if rot is None else rot.freq.data_ptr(), rot_gain=1.0 if rot is None else rot.gain, eps=s.eps, positions=st.positions.data_ptr(),
                             batch_idx=st.batch_idx.data_ptr(), page_table=st.page_table.data_ptr(), pt_stride=st.page_table.stride(0),
                             page_size=st.page_size, k_cache=k_cache.data_ptr(), v_cache=v_cache.data_ptr(), num_slots=k_cache.shape[0],
                             q_out=q.data_ptr(), guard=tcgen05.error_flag(proj.device).data_ptr() + 16)
        N.call("sl_grouped_pre", C.byref(p), T, int(proj.dtype == torch.float32), int(dtype == torch.float32), N.stream())
        return q
    turn = (lambda y: y) if rot is None else (lambda y: rot.apply(y, st.positions))
    x = proj.to(torch.float32)
    if w.bias is not None:
        x = x + w.bias
    if s.kv_heads:
        k = x[:, kb:vb].reshape(T, s.kv_heads, s.dim)
        v = x[:, vb:vb + nv * s.vdim].reshape(T, nv, s.vdim) if s.own_values else k
        slots = _slots(st.positions, st.batch_idx, st.page_table, st.page_size)
        k_cache[slots] = turn(_rms(k, w.k_norm, s.eps)).to(k_cache.dtype)
        v_cache[slots] = v.to(v_cache.dtype)
    return turn(_rms(x[:, :kb].reshape(T, s.heads, s.dim), w.q_norm, s.eps)).to(dtype)


@dataclass
class RowNormWeights:
    """Of :func:`grouped_row_pre`, all fp32; rows are in the adjacent order of `ops/rotary.py`."""

    q_norm: torch.Tensor                    # [heads * dim]
    k_norm: torch.Tensor                    # [kv_heads * dim]
    bias: Optional[torch.Tensor] = None     # [heads * dim | kv_heads * dim | kv_heads * vdim], added to the projection
    gain: Optional[torch.Tensor] = None     # [heads]: factor on a head's scores
    sink: Optional[torch.Tensor] = None


def _turn_at(angles: torch.Tensor, turn: Optional[Turn]) -> int:
    return 0 if turn is None else angles.data_ptr() + turn.at * 8


def grouped_row_pre(proj: torch.Tensor, s: GroupedShape, w: RowNormWeights, turn: Turn, v_turn: Optional[Turn], angles: torch.Tensor, st,
                    k_cache: torch.Tensor, v_cache: torch.Tensor, dtype: torch.dtype, comm=None) -> torch.Tensor:
    """:func:`grouped_pre` with one RMS norm over all heads' queries and one over all heads' keys.  proj [T, q | k | v] (`dtype` or
    fp32), without the biases; queries and keys turn by `turn`, values by `v_turn` (None: they do not).  With several ranks the sums
    of squares are completed by `comm`.  Returns the queries [T, heads, dim]."""
    T, kb = proj.shape[0], s.heads * s.dim
    vb, world = kb + s.kv_heads * s.dim, 1 if comm is None else comm.ctx.world
    if proj.is_cuda:
        N = _native()
        from . import tcgen05
        q = torch.empty(T, s.heads, s.dim, dtype=dtype, device=proj.device)
        at = lambda i: proj.data_ptr() + i * proj.element_size()
        bias = lambda i: 0 if w.bias is None else w.bias.data_ptr() + 4 * i
        p = GroupedRowPreParams(q=at(0), k=at(kb), v=at(vb), ld=proj.stride(0), heads=s.heads, kv_heads=s.kv_heads, dim=s.dim, vdim=s.vdim,
                                rot_dims=turn.dims, q_bias=bias(0), k_bias=bias(kb), v_bias=bias(vb), q_norm=w.q_norm.data_ptr(),
                                k_norm=w.k_norm.data_ptr(), q_count=world * kb, k_count=world * (vb - kb), eps=s.eps, gain=N.ptr(w.gain),
                                qk_turn=_turn_at(angles, turn), v_turn=_turn_at(angles, v_turn), ldt=angles.shape[1],
                                positions=st.positions.data_ptr(), batch_idx=st.batch_idx.data_ptr(), page_table=st.page_table.data_ptr(),
                                pt_stride=st.page_table.stride(0), page_size=st.page_size, k_cache=k_cache.data_ptr(),
                                v_cache=v_cache.data_ptr(), num_slots=k_cache.shape[0], q_out=q.data_ptr(),
                                guard=tcgen05.error_flag(proj.device).data_ptr() + 16)
        in_f32 = int(proj.dtype == torch.float32)
        if world > 1:
            sums = torch.empty(T, 2, dtype=torch.float32, device=proj.device)
            N.call("sl_grouped_row_sums", C.byref(p), sums.data_ptr(), T, in_f32, N.stream())
            sums = comm.all_reduce(sums)
            p.sums = sums.data_ptr()
        N.call("sl_grouped_row_pre", C.byref(p), T, in_f32, int(dtype == torch.float32), N.stream())
        return q
    x = proj[:, :vb + s.kv_heads * s.vdim].to(torch.float32)
    if w.bias is not None:
        x = x + w.bias
    sums = torch.stack([x[:, :kb].square().sum(-1), x[:, kb:vb].square().sum(-1)], -1)
    if world > 1:
        sums = comm.all_reduce(sums)
    q = x[:, :kb] / torch.sqrt(sums[:, :1] / (world * kb) + s.eps) * w.q_norm
    k = x[:, kb:vb] / torch.sqrt(sums[:, 1:] / (world * (vb - kb)) + s.eps) * w.k_norm
    v = x[:, vb:].reshape(T, s.kv_heads, s.vdim)
    q = q.reshape(T, s.heads, s.dim)
    if w.gain is not None:
        q = q * w.gain[:, None]
    slots = _slots(st.positions, st.batch_idx, st.page_table, st.page_size)
    k_cache[slots] = turn.apply(k.reshape(T, s.kv_heads, s.dim), angles).to(k_cache.dtype)
    v_cache[slots] = (v if v_turn is None else v_turn.apply(v, angles)).to(v_cache.dtype)
    return turn.apply(q, angles).to(dtype)


def visible_keys(pos: int, window: int, keep_first: int) -> torch.Tensor:
    """Positions that a query at `pos` sees, in order."""
    first = max(0, pos - window + 1) if window else 0
    return torch.cat([torch.arange(min(keep_first, first)), torch.arange(first, pos + 1)])


@dataclass
class Finish:
    """What happens to a row's sum over the values before it is stored: pairs turned back by the query's angles, a factor."""

    turn: Optional[Turn] = None
    angles: Optional[torch.Tensor] = None
    scale: float = 1.0

    @property
    def kernel_args(self) -> dict:
        return dict(turn=_turn_at(self.angles, self.turn), ldt=0 if self.turn is None else self.angles.shape[1], out_scale=self.scale)


PLAIN = Finish()


def _params(q, s, w, st, k_cache, v_cache, out, finish) -> GroupedAttnParams:
    N = _native()
    from . import tcgen05
    return GroupedAttnParams(q=q.data_ptr(), k_cache=k_cache.data_ptr(), v_cache=v_cache.data_ptr(), num_slots=k_cache.shape[0],
                             positions=st.positions.data_ptr(), batch_idx=st.batch_idx.data_ptr(), page_table=st.page_table.data_ptr(),
                             pt_stride=st.page_table.stride(0), page_size=st.page_size, heads=s.heads, kv_heads=s.kv_heads, dim=s.dim,
                             vdim=s.vdim, window=s.window, keep_first=s.keep_first, splits=1, scale=s.scale, sink=N.ptr(w.sink),
                             out=out.data_ptr(), ldo=out.stride(0), guard=tcgen05.error_flag(q.device).data_ptr() + 16, **finish.kernel_args)


def grouped_attention(q: torch.Tensor, s: GroupedShape, w, st, k_cache, v_cache, out: torch.Tensor, finish: Finish = PLAIN) -> None:
    """Attention of every token row over the cached keys it sees, into `out` [T, heads * vdim] (rows of any stride)."""
    T = q.shape[0]
    if q.is_cuda:
        N = _native()
        mma = q.dtype == torch.bfloat16 and out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0 and s.kv_heads * s.dim % 8 == 0
        if mma and "spans" in st.extra and N.fn("sl_portion_attn_ok")(s.dim, 0, s.vdim):
            return grouped_portions(q, s, w, st, k_cache, v_cache, out, finish)
        if mma and "spans" not in st.extra and N.fn("sl_grouped_decode_ok")(s.dim, s.vdim):
            return grouped_decode(q, s, w, st, k_cache, v_cache, out, finish)
        N.call("sl_grouped_rows", C.byref(_params(q, s, w, st, k_cache, v_cache, out, finish)), T, int(q.dtype == torch.float32), N.stream())
        return
    g = s.heads // s.kv_heads
    for t in range(T):
        kp = visible_keys(int(st.positions[t]), s.window, s.keep_first)
        slots = _slots(kp, torch.full_like(kp, int(st.batch_idx[t])), st.page_table, st.page_size)
        k, v = (c[slots].to(torch.float32).repeat_interleave(g, 1) for c in (k_cache, v_cache))
        sc = torch.einsum("hd,khd->hk", q[t].to(torch.float32), k) * s.scale
        if w.sink is not None:
            sc = torch.cat([sc, w.sink.view(-1, 1)], -1)
        p = torch.softmax(sc, -1)[:, :kp.numel()]
        o = torch.einsum("hk,khv->hv", p, v) * finish.scale
        if finish.turn is not None:
            o = finish.turn.apply(o[None], finish.angles[t:t + 1], back=True)
        out[t] = o.reshape(-1).to(out.dtype)


def grouped_portions(q, s: GroupedShape, w, st, k_cache, v_cache, out, finish: Finish = PLAIN) -> None:
    """Portions of prompts: the rows that the step's windows can see are copied out of the pages, one kernel attends."""
    plan = PortionPlan.of(st, s.window, s.keep_first)
    k = gather_rows(k_cache.view(-1, s.kv_heads * s.dim), plan, st)
    v = gather_rows(v_cache.view(-1, s.kv_heads * s.vdim), plan, st)
    portion_attention(q.view(q.shape[0], -1), s.dim, None, k, v, plan, out, heads=s.heads, h0=0, group=s.heads, dim=s.dim, vdim=s.vdim,
                      kv_group=s.heads // s.kv_heads, window=s.window, keep_first=s.keep_first, scale=s.scale, sink=w.sink, finish=finish.kernel_args)


DECODE_TILE = 64


def decode_splits(T: int, s: GroupedShape, max_kv_len: int) -> int:
    """Key splits of the decode kernel: about three CTAs per SM, at least one tile of keys each."""
    keys = min(s.window + s.keep_first, max_kv_len) if s.window else max_kv_len
    ctas = T * s.kv_heads * -(-(s.heads // s.kv_heads) // 16)
    return max(1, min(-(-444 // ctas), -(-max(1, keys) // DECODE_TILE), 64))


def grouped_decode(q, s: GroupedShape, w, st, k_cache, v_cache, out, finish: Finish = PLAIN) -> None:
    """One query token per page-table row; the keys of a row are shared by several CTAs whose results a second kernel merges."""
    N = _native()
    T, dev = q.shape[0], q.device
    p = _params(q, s, w, st, k_cache, v_cache, out, finish)
    p.splits = decode_splits(T, s, st.max_kv_len)
    if p.splits > 1:
        o_part = torch.empty(T, s.heads, p.splits, s.vdim, dtype=torch.float32, device=dev)
        lse = torch.empty(T, s.heads, p.splits, dtype=torch.float32, device=dev)
        p.o_part, p.lse_part = o_part.data_ptr(), lse.data_ptr()
    N.call("sl_grouped_decode", C.byref(p), T, N.stream())
