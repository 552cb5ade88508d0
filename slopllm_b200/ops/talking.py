"""Talking heads: grouped-query attention over a paged cache in which the scores of all query heads are mixed before the softmax,

    score[h, j] = sum_g talk[h, g] * scale * q_g . k_j[kv(g)],        o_h = softmax_j(score[h, j]) . v_j[kv(h)],

queries and keys normalised per head, with biases on all projections.  Positions may be limited to their own chunk: i sees j <= i if both
lie in the same run of `chunk` positions, counted from the sequence's start.  Mixing needs every head's scores, so a rank that shares
the heads with others has all query and key heads but its own value and output heads only.

CUDA tensors run `csrc/talking_attn.cu` (row preparation: `csrc/grouped_attn.cu`); CPU tensors run the fp32 definition below.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

import torch

from .dense import _slots
from .grouped import GroupedShape, GroupedWeights, grouped_pre


def _native():
    from . import native as N
    return N


class TalkingParams(C.Structure):
    _fields_ = [("q", C.c_void_p), ("k_cache", C.c_void_p), ("v_cache", C.c_void_p), ("num_slots", C.c_int), ("positions", C.c_void_p),
                ("batch_idx", C.c_void_p), ("page_table", C.c_void_p), ("pt_stride", C.c_int), ("page_size", C.c_int), ("heads", C.c_int),
                ("kv_heads", C.c_int), ("out_heads", C.c_int), ("v_heads", C.c_int), ("dim", C.c_int), ("vdim", C.c_int), ("chunk", C.c_int),
                ("scale", C.c_float), ("talk", C.c_void_p), ("out", C.c_void_p), ("ldo", C.c_int), ("guard", C.c_void_p)]


@dataclass
class TalkingShape:
    heads: int                 # query heads whose scores are mixed (all of the layer's)
    kv_heads: int              # their key heads
    out_heads: int             # heads of this rank's output
    v_heads: int               # value heads of this rank
    dim: int
    vdim: int
    scale: float
    chunk: int = 0             # positions of a chunk; 0: the whole sequence is one
    eps: float = 1e-5
    own_kv: bool = True        # False: keys and values are another layer's


@dataclass
class TalkingWeights:
    bias: torch.Tensor         # fp32, of the projection rows q (| k | v)
    talk: torch.Tensor         # fp32 [out_heads, heads]
    ones: torch.Tensor         # fp32 [dim]: the norms have no weight


def first_visible(pos: int, chunk: int) -> int:
    return pos // chunk * chunk if chunk else 0


def talking_pre(proj: torch.Tensor, s: TalkingShape, w: TalkingWeights, st, k_cache: torch.Tensor, v_cache: torch.Tensor, dtype: torch.dtype) -> torch.Tensor:
    """proj [T, heads * dim (q) | kv_heads * dim (k) | v_heads * vdim (v)] (`dtype` or fp32; q alone without keys of its own), without the
    biases: writes normalised keys and values into their slots and returns the normalised queries [T, heads, dim]."""
    kv, v = (s.kv_heads, s.v_heads) if s.own_kv else (0, 0)
    shape = GroupedShape(s.heads, kv, s.dim, s.vdim, s.scale, eps=s.eps, v_heads=v)
    return grouped_pre(proj, shape, GroupedWeights(w.ones, w.ones, bias=w.bias), None, st, k_cache, v_cache, dtype)


def talking_attention(q: torch.Tensor, s: TalkingShape, w: TalkingWeights, st, k_cache, v_cache, out: torch.Tensor) -> None:
    """Attention of every token row over the cached keys it sees, into `out` [T, out_heads * vdim] (rows of any stride)."""
    T = q.shape[0]
    if q.is_cuda:
        N = _native()
        from . import tcgen05
        p = TalkingParams(q=q.data_ptr(), k_cache=k_cache.data_ptr(), v_cache=v_cache.data_ptr(), num_slots=k_cache.shape[0],
                          positions=st.positions.data_ptr(), batch_idx=st.batch_idx.data_ptr(), page_table=st.page_table.data_ptr(),
                          pt_stride=st.page_table.stride(0), page_size=st.page_size, heads=s.heads, kv_heads=s.kv_heads, out_heads=s.out_heads,
                          v_heads=s.v_heads, dim=s.dim, vdim=s.vdim, chunk=s.chunk, scale=s.scale, talk=w.talk.data_ptr(), out=out.data_ptr(),
                          ldo=out.stride(0), guard=tcgen05.error_flag(q.device).data_ptr() + 16)
        N.call("sl_talking_rows", C.byref(p), T, int(q.dtype == torch.float32), N.stream())
        return
    for t in range(T):
        pos = int(st.positions[t])
        kp = torch.arange(first_visible(pos, s.chunk), pos + 1)
        slots = _slots(kp, torch.full_like(kp, int(st.batch_idx[t])), st.page_table, st.page_size)
        k = k_cache[slots].to(torch.float32).repeat_interleave(s.heads // s.kv_heads, 1)
        v = v_cache[slots].to(torch.float32).repeat_interleave(s.out_heads // s.v_heads, 1)
        sc = w.talk @ (torch.einsum("hd,khd->hk", q[t].to(torch.float32), k) * s.scale)
        out[t] = torch.einsum("hk,khv->hv", torch.softmax(sc, -1), v).reshape(-1).to(out.dtype)
