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


class LatentPrefillParams(C.Structure):
    _fields_ = [("q", C.c_void_p), ("ldq", C.c_int), ("q_head", C.c_int), ("q_rot", C.c_void_p), ("k", C.c_void_p), ("ldk", C.c_int),
                ("v", C.c_void_p), ("ldv", C.c_int), ("rows", C.c_void_p), ("row", C.c_int), ("rank", C.c_int), ("tiles", C.c_void_p),
                ("heads", C.c_int), ("h0", C.c_int), ("dim", C.c_int), ("rot_dim", C.c_int), ("vdim", C.c_int), ("window", C.c_int),
                ("scale", C.c_float), ("sink", C.c_void_p), ("out", C.c_void_p), ("err", C.c_void_p), ("stages", C.c_int)]


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


def head_product(x: torch.Tensor, x_head: int, w: torch.Tensor, ops) -> torch.Tensor:
    """out[t, h * n + j] = sum_k x[t, h * x_head + k] w[h, k, j] for every head (w [heads, K, n])."""
    N = _native()
    T, (h, K, n) = x.shape[0], w.shape
    if w.dtype == torch.bfloat16 and x.stride(0) % 8 == 0 and n % 8 == 0 and x_head % 8 == 0:
        if T > 32:
            out = ops._head_batched_gemm(x, x_head, K, None, w)
            if out is not None:
                return out
        out = torch.empty(T, h * n, dtype=torch.bfloat16, device=x.device)
        N.call("sl_bmv", out.data_ptr(), x.data_ptr(), w.data_ptr(), T, h, K, n, x.stride(0), x_head, 0, 0, N.stream())
        return out
    out = torch.empty(T, h * n, dtype=w.dtype, device=x.device)
    p = N.SimtLinearParams(y=out.data_ptr(), x=x.data_ptr(), w=w.data_ptr(), T=T, N=n, K=K, batch=h, y_t=h * n, y_b=n, x_t=x.stride(0),
                           x_b=x_head, w_n=1, w_k=n, w_b=K * n)
    N.call("sl_linear_simt", C.byref(p), int(w.dtype == torch.float32), int(w.dtype == torch.float32), N.stream())
    return out


def latent_attention(qd: torch.Tensor, q_rot: torch.Tensor, s: LatentShape, w: LatentWeights, st, cache: torch.Tensor, ops=None) -> torch.Tensor:
    """Attention of every token row over the cached rows of its sequence that its window shows.  The unrotated queries are
    read from the projection rows `qd`.  Returns [T, heads * vdim]."""
    T, qs = qd.shape[0], s.dim + s.rot_dim
    if qd.is_cuda:
        N = _native()
        mma = qd.dtype == torch.bfloat16 and qd.stride(0) % 8 == 0 and N.fn("sl_latent_mma_ok")(s.dim, s.rot_dim, s.vdim, s.rank)
        if mma and "spans" in st.extra:
            return latent_prefill(qd, q_rot, s, w, st, cache, ops)
        q_abs = head_product(qd, qs, w.uk, ops)
        if mma:
            return latent_decode(q_abs, q_rot, s, w, st, cache, ops)
        o = latent_rows(q_abs, q_rot, s, w, st, cache)
        return head_product(o.view(T, s.heads * s.rank), s.rank, w.uv_t, ops)
    q = qd[:, :s.heads * qs].reshape(T, s.heads, qs)[..., :s.dim].to(torch.float32)
    out = torch.empty(T, s.heads, s.vdim, dtype=torch.float32)
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
        out[t] = torch.einsum("hvr,hr->hv", w.uv.to(torch.float32), p @ c)
    return out.reshape(T, s.heads * s.vdim).to(qd.dtype)


class PortionPlan:
    """Key ranges and query tiles of a step's portions for one window size, on the device."""

    def __init__(self, spans, window: int, device):
        ranges, tiles = [], []
        row = tok = 0
        for b, (start, n) in enumerate(spans):
            lo = max(0, start - window + 1) if window else 0
            ranges.append((b, lo, start + n - lo, row))
            tiles += [(tok + o, min(QUERY_TILE, n - o), start + o, row - lo) for o in range(0, n, QUERY_TILE)]
            row += start + n - lo
            tok += n
        self.batch, self.tile_count, self.rows, self.longest = len(ranges), len(tiles), row, max(r[2] for r in ranges)
        t = torch.tensor([x for r in ranges + tiles for x in r], dtype=torch.int32, device=device)
        self.ranges, self.tiles = t[:4 * self.batch], t[4 * self.batch:]

    @staticmethod
    def of(st, window: int) -> "PortionPlan":
        plans = st.extra.setdefault("portion_plans", {})
        if window not in plans:
            plans[window] = PortionPlan(st.extra["spans"], window, st.input_ids.device)
        return plans[window]


def latent_prefill(qd, q_rot, s: LatentShape, w: LatentWeights, st, cache, ops) -> torch.Tensor:
    """Expanded attention of a step's portions: the visible cache rows are copied out of the pages, two GEMMs make the heads'
    keys and values, one kernel attends."""
    from ..models.weights import LinearWeight
    N = _native()
    from . import tcgen05
    T, dev = qd.shape[0], qd.device
    plan = PortionPlan.of(st, s.window)
    rows = torch.empty(plan.rows, s.row, dtype=torch.bfloat16, device=dev)
    gp = LatentGatherParams(out=rows.data_ptr(), cache=cache.data_ptr(), num_slots=cache.shape[0], row=s.row, ranges=plan.ranges.data_ptr(),
                            page_table=st.page_table.data_ptr(), pt_stride=st.page_table.stride(0), page_size=st.page_size,
                            guard=tcgen05.error_flag(dev).data_ptr() + 16)
    N.call("sl_latent_gather", C.byref(gp), plan.batch, plan.longest, N.stream())
    out = torch.empty(T, s.heads * s.vdim, dtype=torch.bfloat16, device=dev)
    group = max(1, min(s.heads, EXPAND_BUDGET_BYTES // (plan.rows * (s.dim + s.vdim) * 2)))
    lat = rows[:, :s.rank]
    uk, uv = w.uk.view(s.heads * s.dim, s.rank), w.uv.view(s.heads * s.vdim, s.rank)
    for h0 in range(0, s.heads, group):
        hn = min(group, s.heads - h0)
        k = ops.linear(lat, LinearWeight(uk[h0 * s.dim:(h0 + hn) * s.dim]))
        v = ops.linear(lat, LinearWeight(uv[h0 * s.vdim:(h0 + hn) * s.vdim]))
        latent_prefill_kernel(qd, q_rot, s, w, rows, k, v, plan, h0, hn, out)
    return out


def latent_prefill_kernel(qd, q_rot, s: LatentShape, w: LatentWeights, rows, k, v, plan: PortionPlan, h0: int, heads: int, out) -> None:
    """Attention of heads h0 .. h0 + heads - 1 over their expanded keys k [rows, heads * dim] and values v [rows, heads * vdim]."""
    N = _native()
    from . import tcgen05
    p = LatentPrefillParams(q=qd.data_ptr(), ldq=qd.stride(0), q_head=s.dim + s.rot_dim, q_rot=q_rot.data_ptr(), k=k.data_ptr(),
                            ldk=k.stride(0), v=v.data_ptr(), ldv=v.stride(0), rows=rows.data_ptr(), row=s.row, rank=s.rank,
                            tiles=plan.tiles.data_ptr(), heads=s.heads, h0=h0, dim=s.dim, rot_dim=s.rot_dim, vdim=s.vdim,
                            window=s.window, scale=s.scale, sink=N.ptr(w.sink), out=out.data_ptr(), err=tcgen05.error_flag(out.device).data_ptr())
    N.call("sl_latent_prefill", C.byref(p), heads, plan.tile_count, N.stream())


def decode_splits(T: int, heads: int, keys: int) -> int:
    """Key splits of the decode kernel: two CTAs per SM, at least one tile of keys each."""
    ctas = T * -(-heads // 16)
    return max(1, min(-(-296 // ctas), -(-keys // KEY_TILE), 64))


def latent_decode(q_abs, q_rot, s: LatentShape, w: LatentWeights, st, cache, ops) -> torch.Tensor:
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
        return head_product(o.view(T, s.heads * s.rank), s.rank, w.uv_t, ops)
    o_part = torch.empty(T, s.heads, splits, s.rank, dtype=torch.float32, device=dev)
    lse = torch.empty(T, s.heads, splits, dtype=torch.float32, device=dev)
    p.o_part, p.lse_part = o_part.data_ptr(), lse.data_ptr()
    N.call("sl_latent_decode", C.byref(p), T, N.stream())
    if fused:
        out = torch.empty(T, s.heads * s.vdim, dtype=torch.bfloat16, device=dev)
        cp = N.CombineExpandParams(o_part=o_part.data_ptr(), lse_part=lse.data_ptr(), w_v=w.uv_t.data_ptr(), y=out.data_ptr(), T=T,
                                   tpad=T, Hh=s.heads, K=s.rank, N=s.vdim, np=splits)
        N.call("sl_combine_vexpand", C.byref(cp), N.stream())
        return out
    o, _ = ops.combine([o_part], [lse], want_lse=False)
    return head_product(o.view(T, s.heads * s.rank), s.rank, w.uv_t, ops)


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
