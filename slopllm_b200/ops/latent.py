"""Latent attention over a paged cache of plain rows [latent | rotated key part] shared by all heads: sliding window, softmax
sink, any rotary table.  CUDA tensors run `csrc/latent_attn.cu`; CPU tensors run the fp32 definition below.

Two forms of the same product: *absorbed* (queries are multiplied by the key expansion, the heads attend over the latent rows
themselves and the result is expanded to values) for decoding, and *expanded* (keys and values of the visible range are
materialised per head) for portions of prompts.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch

from .dense import _slots
from .rotary import RotaryTable


def _native():
    from . import native as N
    return N


class LatentPreParams(C.Structure):
    _fields_ = [("qd", C.c_void_p), ("ld", C.c_int), ("heads", C.c_int), ("dim", C.c_int), ("rot_dim", C.c_int), ("rot_dims", C.c_int),
                ("rank", C.c_int), ("norm_w", C.c_void_p), ("freq", C.c_void_p), ("rot_gain", C.c_float), ("eps", C.c_float),
                ("positions", C.c_void_p), ("batch_idx", C.c_void_p), ("page_table", C.c_void_p), ("pt_stride", C.c_int),
                ("page_size", C.c_int), ("cache", C.c_void_p), ("num_slots", C.c_int), ("q_rot", C.c_void_p), ("guard", C.c_void_p)]


class LatentRowsParams(C.Structure):
    _fields_ = [("q_abs", C.c_void_p), ("q_rot", C.c_void_p), ("cache", C.c_void_p), ("num_slots", C.c_int), ("positions", C.c_void_p),
                ("batch_idx", C.c_void_p), ("page_table", C.c_void_p), ("pt_stride", C.c_int), ("page_size", C.c_int), ("heads", C.c_int),
                ("rank", C.c_int), ("rot_dim", C.c_int), ("window", C.c_int), ("scale", C.c_float), ("sink", C.c_void_p),
                ("out", C.c_void_p), ("guard", C.c_void_p)]


class LatentGatherParams(C.Structure):
    _fields_ = [("out", C.c_void_p), ("cache", C.c_void_p), ("num_slots", C.c_int), ("row", C.c_int), ("ranges", C.c_void_p),
                ("page_table", C.c_void_p), ("pt_stride", C.c_int), ("page_size", C.c_int), ("guard", C.c_void_p)]


class PortionAttnParams(C.Structure):
    _fields_ = [("q", C.c_void_p), ("ldq", C.c_int), ("q_head", C.c_int), ("q_rot", C.c_void_p), ("k", C.c_void_p), ("ldk", C.c_int),
                ("v", C.c_void_p), ("ldv", C.c_int), ("rows", C.c_void_p), ("row", C.c_int), ("rank", C.c_int), ("tiles", C.c_void_p),
                ("heads", C.c_int), ("h0", C.c_int), ("dim", C.c_int), ("rot_dim", C.c_int), ("vdim", C.c_int), ("kv_group", C.c_int),
                ("window", C.c_int), ("keep_first", C.c_int), ("scale", C.c_float), ("sink", C.c_void_p), ("out", C.c_void_p),
                ("ldo", C.c_int), ("err", C.c_void_p), ("stages", C.c_int), ("turn", C.c_void_p), ("ldt", C.c_int), ("out_scale", C.c_float)]


class LatentDecodeParams(C.Structure):
    _fields_ = [("q_abs", C.c_void_p), ("q_rot", C.c_void_p), ("cache", C.c_void_p), ("num_slots", C.c_int), ("positions", C.c_void_p),
                ("batch_idx", C.c_void_p), ("page_table", C.c_void_p), ("pt_stride", C.c_int), ("page_size", C.c_int), ("heads", C.c_int),
                ("rank", C.c_int), ("rot_dim", C.c_int), ("window", C.c_int), ("splits", C.c_int), ("scale", C.c_float),
                ("sink", C.c_void_p), ("o_part", C.c_void_p), ("lse_part", C.c_void_p), ("o_final", C.c_void_p), ("guard", C.c_void_p)]


EXPAND_BUDGET_BYTES = 1 << 30      # transient keys + values of the expanded form; more goes in groups of heads
QUERY_TILE, KEY_TILE = 128, 64     # of the tensor-core kernels (csrc/latent_mma.cu)


@dataclass
class LatentShape:
    heads: int                 # heads of this rank
    dim: int                   # unrotated query / key values per head
    rot_dim: int               # rotated ones
    vdim: int
    rank: int
    scale: float
    window: int = 0            # a position sees itself and window - 1 tokens before it; 0: all of them
    eps: float = 1e-5

    @property
    def row(self) -> int:
        return self.rank + self.rot_dim


@dataclass
class LatentWeights:
    norm: torch.Tensor                      # fp32 [rank], weight of the latent's RMS norm
    uk: torch.Tensor                        # [heads, dim, rank]
    uv: torch.Tensor                        # [heads, vdim, rank]
    uv_t: torch.Tensor                      # [heads, rank, vdim]: the same, for the value expansion of decoded rows
    sink: Optional[torch.Tensor] = None     # fp32 [heads]


def latent_pre(qd: torch.Tensor, s: LatentShape, w: LatentWeights, rot: RotaryTable, st, cache: torch.Tensor) -> torch.Tensor:
    """qd [T, heads * (dim + rot_dim) | rank | rot_dim]: normalises the latent, rotates the shared key part and writes the
    cache row; returns the rotated query parts [T, heads, rot_dim]."""
    T = qd.shape[0]
    if qd.is_cuda:
        N = _native()
        from . import tcgen05
        q_rot = torch.empty(T, s.heads, s.rot_dim, dtype=qd.dtype, device=qd.device)
        p = LatentPreParams(qd=qd.data_ptr(), ld=qd.stride(0), heads=s.heads, dim=s.dim, rot_dim=s.rot_dim, rot_dims=rot.dims,
                            rank=s.rank, norm_w=w.norm.data_ptr(), freq=rot.freq.data_ptr(), rot_gain=rot.gain, eps=s.eps,
                            positions=st.positions.data_ptr(), batch_idx=st.batch_idx.data_ptr(), page_table=st.page_table.data_ptr(),
                            pt_stride=st.page_table.stride(0), page_size=st.page_size, cache=cache.data_ptr(), num_slots=cache.shape[0],
                            q_rot=q_rot.data_ptr(), guard=tcgen05.error_flag(qd.device).data_ptr() + 16)
        N.call("sl_latent_pre", C.byref(p), T, int(qd.dtype == torch.float32), N.stream())
        return q_rot
    qs = s.dim + s.rot_dim
    lat = qd[:, s.heads * qs:s.heads * qs + s.rank].to(torch.float32)
    lat = lat / torch.sqrt((lat * lat).mean(-1, keepdim=True) + s.eps) * w.norm
    k_rot = rot.apply(qd[:, s.heads * qs + s.rank:], st.positions)
    cache[_slots(st.positions, st.batch_idx, st.page_table, st.page_size)] = torch.cat([lat, k_rot], -1).to(cache.dtype)
    return rot.apply(qd[:, :s.heads * qs].reshape(T, s.heads, qs)[..., s.dim:], st.positions).to(qd.dtype)


def head_product(x: torch.Tensor, x_head: int, w: torch.Tensor, ops, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """out[t, h * n + j] = sum_k x[t, h * x_head + k] w[h, k, j] for every head (w [heads, K, n]); `out`: rows of any stride."""
    N = _native()
    T, (h, K, n) = x.shape[0], w.shape
    if w.dtype == torch.bfloat16 and x.stride(0) % 8 == 0 and n % 8 == 0 and x_head % 8 == 0 and (out is None or out.stride(0) % 8 == 0):
        if T > 32:
            o = ops._head_batched_gemm(x, x_head, K, None, w, out)
            if o is not None:
                return o
        if out is None or out.is_contiguous():
            out = torch.empty(T, h * n, dtype=torch.bfloat16, device=x.device) if out is None else out
            N.call("sl_bmv", out.data_ptr(), x.data_ptr(), w.data_ptr(), T, h, K, n, x.stride(0), x_head, 0, 0, N.stream())
            return out
    out = torch.empty(T, h * n, dtype=w.dtype, device=x.device) if out is None else out
    p = N.SimtLinearParams(y=out.data_ptr(), x=x.data_ptr(), w=w.data_ptr(), T=T, N=n, K=K, batch=h, y_t=out.stride(0), y_b=n, x_t=x.stride(0),
                           x_b=x_head, w_n=1, w_k=n, w_b=K * n)
    N.call("sl_linear_simt", C.byref(p), int(w.dtype == torch.float32), int(w.dtype == torch.float32), N.stream())
    return out


def latent_attention(qd: torch.Tensor, q_rot: torch.Tensor, s: LatentShape, w: LatentWeights, st, cache: torch.Tensor, ops=None,
                     out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Attention of every token row over the cached rows of its sequence that its window shows.  The unrotated queries are
    read from the projection rows `qd`.  Returns [T, heads * vdim] (`out`, rows of any stride, when given)."""
    T, qs = qd.shape[0], s.dim + s.rot_dim
    if out is None:
        out = torch.empty(T, s.heads * s.vdim, dtype=qd.dtype, device=qd.device)
    if qd.is_cuda:
        N = _native()
        mma = (qd.dtype == torch.bfloat16 and qd.stride(0) % 8 == 0 and qd.data_ptr() % 16 == 0 and out.stride(0) % 8 == 0
               and N.fn("sl_latent_mma_ok")(s.dim, s.rot_dim, s.vdim, s.rank))
        if mma and "spans" in st.extra:
            return latent_prefill(qd, q_rot, s, w, st, cache, ops, out)
        q_abs = head_product(qd, qs, w.uk, ops)
        if mma:
            return latent_decode(q_abs, q_rot, s, w, st, cache, ops, out)
        o = latent_rows(q_abs, q_rot, s, w, st, cache)
        return head_product(o.view(T, s.heads * s.rank), s.rank, w.uv_t, ops, out)
    q = qd[:, :s.heads * qs].reshape(T, s.heads, qs)[..., :s.dim].to(torch.float32)
    for t in range(T):
        pos = int(st.positions[t])
        kp = torch.arange(max(0, pos - s.window + 1) if s.window else 0, pos + 1)
        rows = cache[_slots(kp, torch.full_like(kp, int(st.batch_idx[t])), st.page_table, st.page_size)].to(torch.float32)
        c, kr = rows[:, :s.rank], rows[:, s.rank:]
        k = torch.einsum("hdr,kr->hkd", w.uk.to(torch.float32), c)
        sc = (torch.einsum("hd,hkd->hk", q[t], k) + q_rot[t].to(torch.float32) @ kr.t()) * s.scale
        if w.sink is not None:
            sc = torch.cat([sc, w.sink.view(-1, 1)], -1)
        p = torch.softmax(sc, -1)[:, :kp.numel()]
        out[t] = torch.einsum("hvr,hr->hv", w.uv.to(torch.float32), p @ c).reshape(-1).to(out.dtype)
    return out


class PortionPlan:
    """Key ranges and query tiles of a step's portions for one window size and number of kept first tokens, on the device.  A
    sequence's visible rows are gathered as its kept rows (those in front of the window) followed by the window's."""

    def __init__(self, spans, window: int, keep_first: int, device):
        ranges, tiles = [], []
        row = tok = 0
        for b, (start, n) in enumerate(spans):
            lo = max(0, start - window + 1) if window else 0
            kept = min(keep_first, lo)
            if kept:
                ranges.append((b, 0, kept, row))
            ranges.append((b, lo, start + n - lo, row + kept))
            tiles += [(tok + o, min(QUERY_TILE, n - o), start + o, row + kept - lo, row) for o in range(0, n, QUERY_TILE)]
            row += kept + start + n - lo
            tok += n
        self.range_count, self.tile_count, self.rows, self.longest = len(ranges), len(tiles), row, max(r[2] for r in ranges)
        t = torch.tensor([x for r in ranges + tiles for x in r], dtype=torch.int32, device=device)
        self.ranges, self.tiles = t[:4 * len(ranges)], t[4 * len(ranges):]

    @staticmethod
    def of(st, window: int, keep_first: int = 0) -> "PortionPlan":
        plans = st.extra.setdefault("portion_plans", {})
        key = (window, keep_first)
        if key not in plans:
            plans[key] = PortionPlan(st.extra["spans"], window, keep_first, st.input_ids.device)
        return plans[key]


def gather_rows(cache: torch.Tensor, plan: PortionPlan, st) -> torch.Tensor:
    """The bf16 cache rows [slots, row] that a step's portions can see, copied out of the pages in the plan's order."""
    N = _native()
    from . import tcgen05
    rows = torch.empty(plan.rows, cache.shape[1], dtype=torch.bfloat16, device=cache.device)
    gp = LatentGatherParams(out=rows.data_ptr(), cache=cache.data_ptr(), num_slots=cache.shape[0], row=cache.shape[1], ranges=plan.ranges.data_ptr(),
                            page_table=st.page_table.data_ptr(), pt_stride=st.page_table.stride(0), page_size=st.page_size,
                            guard=tcgen05.error_flag(cache.device).data_ptr() + 16)
    N.call("sl_latent_gather", C.byref(gp), plan.range_count, plan.longest, N.stream())
    return rows


def portion_attention(q, q_head: int, q_rot, k, v, plan: PortionPlan, out, *, heads: int, h0: int, group: int, dim: int, vdim: int,
                      scale: float, sink=None, kv_group: int = 1, window: int = 0, keep_first: int = 0, rot_dim: int = 0, rows=None,
                      rank: int = 0, finish: Optional[dict] = None) -> None:
    """Attention of heads h0 .. h0 + group - 1 over gathered keys k and values v [rows, ...], into `out` (rows of any stride).
    `finish`: kernel arguments of a rotation and factor on the output (`ops/grouped.py: Finish`)."""
    N = _native()
    from . import tcgen05
    p = PortionAttnParams(q=q.data_ptr(), ldq=q.stride(0), q_head=q_head, q_rot=N.ptr(q_rot), k=k.data_ptr(), ldk=k.stride(0),
                          v=v.data_ptr(), ldv=v.stride(0), rows=N.ptr(rows), row=0 if rows is None else rows.shape[1], rank=rank,
                          tiles=plan.tiles.data_ptr(), heads=heads, h0=h0, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_group=kv_group,
                          window=window, keep_first=keep_first, scale=scale, sink=N.ptr(sink), out=out.data_ptr(), ldo=out.stride(0),
                          err=tcgen05.error_flag(out.device).data_ptr(), **(finish or dict(out_scale=1.0)))
    N.call("sl_portion_attn", C.byref(p), group, plan.tile_count, N.stream())


def latent_prefill(qd, q_rot, s: LatentShape, w: LatentWeights, st, cache, ops, out) -> torch.Tensor:
    """Expanded attention of a step's portions: the visible cache rows are copied out of the pages, two GEMMs make the heads'
    keys and values, one kernel attends."""
    from ..models.weights import LinearWeight
    plan = PortionPlan.of(st, s.window)
    rows = gather_rows(cache, plan, st)
    group = max(1, min(s.heads, EXPAND_BUDGET_BYTES // (plan.rows * (s.dim + s.vdim) * 2)))
    lat = rows[:, :s.rank]
    uk, uv = w.uk.view(s.heads * s.dim, s.rank), w.uv.view(s.heads * s.vdim, s.rank)
    for h0 in range(0, s.heads, group):
        hn = min(group, s.heads - h0)
        k = ops.linear(lat, LinearWeight(uk[h0 * s.dim:(h0 + hn) * s.dim]))
        v = ops.linear(lat, LinearWeight(uv[h0 * s.vdim:(h0 + hn) * s.vdim]))
        portion_attention(qd, s.dim + s.rot_dim, q_rot, k, v, plan, out, heads=s.heads, h0=h0, group=hn, dim=s.dim, vdim=s.vdim,
                          window=s.window, scale=s.scale, sink=w.sink, rot_dim=s.rot_dim, rows=rows, rank=s.rank)
    return out


def decode_splits(T: int, heads: int, keys: int) -> int:
    """Key splits of the decode kernel: two CTAs per SM, at least one tile of keys each."""
    ctas = T * -(-heads // 16)
    return max(1, min(-(-296 // ctas), -(-keys // KEY_TILE), 64))


def latent_decode(q_abs, q_rot, s: LatentShape, w: LatentWeights, st, cache, ops, out) -> torch.Tensor:
    """Absorbed attention of one query token per page-table row and the value expansion -> [T, heads * vdim]."""
    N = _native()
    from . import tcgen05
    T, dev = q_rot.shape[0], q_rot.device
    keys = min(s.window, st.max_kv_len) if s.window else st.max_kv_len
    splits = decode_splits(T, s.heads, max(1, keys))
    fused = T <= 32 and s.vdim % 8 == 0 and s.rank % 4 == 0       # merge of the splits inside the value expansion
    p = LatentDecodeParams(q_abs=q_abs.data_ptr(), q_rot=q_rot.data_ptr(), cache=cache.data_ptr(), num_slots=cache.shape[0],
                           positions=st.positions.data_ptr(), batch_idx=st.batch_idx.data_ptr(), page_table=st.page_table.data_ptr(),
                           pt_stride=st.page_table.stride(0), page_size=st.page_size, heads=s.heads, rank=s.rank, rot_dim=s.rot_dim,
                           window=s.window, splits=splits, scale=s.scale, sink=N.ptr(w.sink), guard=tcgen05.error_flag(dev).data_ptr() + 16)
    if splits == 1 and not fused:
        o = torch.empty(T, s.heads, s.rank, dtype=torch.bfloat16, device=dev)
        p.o_final = o.data_ptr()
        N.call("sl_latent_decode", C.byref(p), T, N.stream())
        return head_product(o.view(T, s.heads * s.rank), s.rank, w.uv_t, ops, out)
    o_part = torch.empty(T, s.heads, splits, s.rank, dtype=torch.float32, device=dev)
    lse = torch.empty(T, s.heads, splits, dtype=torch.float32, device=dev)
    p.o_part, p.lse_part = o_part.data_ptr(), lse.data_ptr()
    N.call("sl_latent_decode", C.byref(p), T, N.stream())
    if fused:
        cp = N.CombineExpandParams(o_part=o_part.data_ptr(), lse_part=lse.data_ptr(), w_v=w.uv_t.data_ptr(), y=out.data_ptr(), T=T,
                                   tpad=T, Hh=s.heads, K=s.rank, N=s.vdim, np=splits, ldy=out.stride(0))
        N.call("sl_combine_vexpand", C.byref(cp), N.stream())
        return out
    o, _ = ops.combine([o_part], [lse], want_lse=False)
    return head_product(o.view(T, s.heads * s.rank), s.rank, w.uv_t, ops, out)


def latent_rows(q_abs, q_rot, s: LatentShape, w: LatentWeights, st, cache) -> torch.Tensor:
    """Absorbed attention of independent token rows -> [T, heads, rank] (any sizes, bf16 or fp32)."""
    N = _native()
    from . import tcgen05
    T = q_rot.shape[0]
    out = torch.empty(T, s.heads, s.rank, dtype=q_rot.dtype, device=q_rot.device)
    p = LatentRowsParams(q_abs=q_abs.data_ptr(), q_rot=q_rot.data_ptr(), cache=cache.data_ptr(), num_slots=cache.shape[0],
                         positions=st.positions.data_ptr(), batch_idx=st.batch_idx.data_ptr(), page_table=st.page_table.data_ptr(),
                         pt_stride=st.page_table.stride(0), page_size=st.page_size, heads=s.heads, rank=s.rank, rot_dim=s.rot_dim,
                         window=s.window, scale=s.scale, sink=N.ptr(w.sink), out=out.data_ptr(),
                         guard=tcgen05.error_flag(q_rot.device).data_ptr() + 16)
    N.call("sl_latent_rows", C.byref(p), T, int(q_rot.dtype == torch.float32), N.stream())
    return out
