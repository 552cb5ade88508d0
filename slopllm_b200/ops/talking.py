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
                ("scale", C.c_float), ("talk", C.c_void_p), ("out", C.c_void_p), ("ldo", C.c_int), ("guard", C.c_void_p),
                ("tiles", C.c_void_p), ("splits", C.c_int), ("o_part", C.c_void_p), ("lse_part", C.c_void_p), ("err", C.c_void_p)]


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


SMS = 148


def key_splits(work: int, keys: int, tile: int) -> int:
    """Blocks that share the keys of each of `work` query tiles (one block per SM at a time): the number with the least tiles of keys one
    after the other, counting one and a half for a block's start and end."""
    tiles = -(-max(1, keys) // tile)
    most = max(1, min(64, tiles, 4 * SMS // work))
    cost = lambda s: -(-work * s // SMS) * (-(-tiles // s) + 1.5) + (1.0 if s > 1 else 0.0)
    return min(range(1, most + 1), key=cost)


class TalkingPlan:
    """Query tiles of a step's portions, those with the most keys first: (first token, tokens, first position, sequence)."""

    def __init__(self, spans, queries: int, chunk: int, device):
        tiles, tok = [], 0
        for b, (start, n) in enumerate(spans):
            tiles += [(tok + o, min(queries, n - o), start + o, b) for o in range(0, n, queries)]
            tok += n
        keys = lambda t: t[2] + t[1] - first_visible(t[2], chunk)
        tiles.sort(key=keys, reverse=True)
        self.count, self.longest = len(tiles), keys(tiles[0])
        self.tiles = torch.tensor(tiles, dtype=torch.int32, device=device)

    @staticmethod
    def of(st, queries: int, chunk: int) -> "TalkingPlan":
        plans = st.extra.setdefault("talking_plans", {})
        if (queries, chunk) not in plans:
            plans[queries, chunk] = TalkingPlan(st.extra["spans"], queries, chunk, st.input_ids.device)
        return plans[queries, chunk]


def talking_attention(q: torch.Tensor, s: TalkingShape, w: TalkingWeights, st, k_cache, v_cache, out: torch.Tensor) -> None:
    """Attention of every token row over the cached keys it sees, into `out` [T, out_heads * vdim] (rows of any stride)."""
    T = q.shape[0]
    if q.is_cuda:
        N = _native()
        from . import tcgen05
        err = tcgen05.error_flag(q.device).data_ptr()
        p = TalkingParams(q=q.data_ptr(), k_cache=k_cache.data_ptr(), v_cache=v_cache.data_ptr(), num_slots=k_cache.shape[0],
                          positions=st.positions.data_ptr(), batch_idx=st.batch_idx.data_ptr(), page_table=st.page_table.data_ptr(),
                          pt_stride=st.page_table.stride(0), page_size=st.page_size, heads=s.heads, kv_heads=s.kv_heads, out_heads=s.out_heads,
                          v_heads=s.v_heads, dim=s.dim, vdim=s.vdim, chunk=s.chunk, scale=s.scale, talk=w.talk.data_ptr(), out=out.data_ptr(),
                          ldo=out.stride(0), guard=err + 16, splits=1, err=err)
        decode = "spans" not in st.extra
        sizes = (s.heads, s.kv_heads, s.out_heads, s.v_heads, s.dim, s.vdim, int(decode))
        queries = N.fn("sl_talking_queries")(*sizes) if q.dtype == torch.bfloat16 and out.stride(0) % 2 == 0 else 0
        if not queries:
            N.call("sl_talking_rows", C.byref(p), T, int(q.dtype == torch.float32), N.stream())
            return
        if decode:
            work, keys = T, min(s.chunk or st.max_kv_len, st.max_kv_len)
        else:
            plan = TalkingPlan.of(st, queries, s.chunk)
            work, keys, p.tiles = plan.count, plan.longest, plan.tiles.data_ptr()
        p.splits = key_splits(work, keys, N.fn("sl_talking_keys")(*sizes))
        if p.splits > 1:
            o_part = torch.empty(T, s.out_heads, p.splits, s.vdim, dtype=torch.float32, device=q.device)
            lse = torch.empty(T, s.out_heads, p.splits, dtype=torch.float32, device=q.device)
            p.o_part, p.lse_part = o_part.data_ptr(), lse.data_ptr()
        N.call("sl_talking_mma", C.byref(p), work, T, N.stream())
        return
    for t in range(T):
        pos = int(st.positions[t])
        kp = torch.arange(first_visible(pos, s.chunk), pos + 1)
        slots = _slots(kp, torch.full_like(kp, int(st.batch_idx[t])), st.page_table, st.page_size)
        k = k_cache[slots].to(torch.float32).repeat_interleave(s.heads // s.kv_heads, 1)
        v = v_cache[slots].to(torch.float32).repeat_interleave(s.out_heads // s.v_heads, 1)
        sc = w.talk @ (torch.einsum("hd,khd->hk", q[t].to(torch.float32), k) * s.scale)
        out[t] = torch.einsum("hk,khv->hv", torch.softmax(sc, -1), v).reshape(-1).to(out.dtype)
