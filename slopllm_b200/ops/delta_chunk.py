"""Chunked form of the channel-wise gated delta rule (`csrc/delta_chunk.cu`): allocation, passes and launches."""
from __future__ import annotations

import ctypes as C

import torch

from .recurrent import CHUNK, CHUNK_MIN_Q, GatedChunkParams, GatedScanParams

SCRATCH_BYTES = 192 << 20           # operands and states of the chunks of one pass; longer steps run in several passes


class DeltaChunkParams(C.Structure):
    _fields_ = [("c", GatedChunkParams), ("dt_bias", C.c_void_p), ("A_log", C.c_void_p), ("beta", C.c_void_p), ("ld_beta", C.c_int),
                ("unit_eps", C.c_float), ("w", C.c_void_p), ("kt", C.c_void_p), ("u0", C.c_void_p), ("u", C.c_void_p),
                ("unit", C.c_void_p), ("stages", C.c_int)]


def usable(s, plan, x, out) -> bool:
    from . import native as N
    return bool(plan is not None and plan.longest >= CHUNK_MIN_Q and x.dtype == torch.bfloat16 and out.dtype == torch.bfloat16
                and x.stride(0) % 8 == 0 and s.kv_heads * s.dk % 8 == 0 and out.stride(0) % 2 == 0 and N.fn("sl_delta_chunk_ok")(s.dk, s.dv))


def run(x, fine, s, w, S, qo_indptr, state_idx, out, ops, plan) -> None:
    """x bf16 [T, q | k | v channels] behind the convolutions, fine fp32 [T, decay rank | gate rank | heads (beta)]."""
    from ..models.weights import LinearWeight
    from . import native as N
    from .delta import UNIT_EPS
    T, h, dk, dv, dev = x.shape[0], s.heads, s.dk, s.dv, x.device
    ra, rg, qk = w.a2.shape[1], w.g2.shape[1], s.kv_heads * dk
    low = fine[:, :ra + rg].to(torch.bfloat16)
    z = ops.linear(low[:, :ra], LinearWeight(w.a2), out_f32=True)
    gate = ops.linear(low[:, ra:], LinearWeight(w.g2))
    if z.stride(0) != h * dk:
        z = z.contiguous()
    per_head = dk * dv * 4 + CHUNK * (2 * dk * 4 + dv * 8)
    per_pass = min(plan.count, max(1, SCRATCH_BYTES // (h * per_head)))
    n = per_pass * h
    e = lambda count, dtype: torch.empty(count, dtype=dtype, device=dev)
    loc, u0, unit = e(n * dk * dv, torch.float32), e(n * CHUNK * dv, torch.float32), e(T * h * 2, torch.float32)
    wb, kt, u = e(n * 2 * CHUNK * dk, torch.bfloat16), e(n * 2 * CHUNK * dk, torch.bfloat16), e(n * 2 * CHUNK * dv, torch.bfloat16)
    at = lambda i: x.data_ptr() + 2 * i
    sp = GatedScanParams(out=out.data_ptr(), q=at(0), k=at(qk), v=at(2 * qk), g=gate.data_ptr(), ld=x.stride(0), norm_w=w.norm.data_ptr(),
                         eps=s.eps, S=S.data_ptr(), qo_indptr=qo_indptr.data_ptr(), state_idx=state_idx.data_ptr(), h=h, dk=dk, dv=dv,
                         ldg=gate.stride(0), ldo=out.stride(0), group=h // s.kv_heads)
    cp = GatedChunkParams(s=sp, chunks=plan.table.data_ptr(), seq_chunks=plan.seq_chunks.data_ptr(), b=z.data_ptr(), loc=loc.data_ptr())
    p = DeltaChunkParams(c=cp, dt_bias=w.dt_bias.data_ptr(), A_log=w.A_log.data_ptr(), beta=fine.data_ptr() + 4 * (ra + rg), ld_beta=fine.stride(0),
                         unit_eps=UNIT_EPS, w=wb.data_ptr(), kt=kt.data_ptr(), u0=u0.data_ptr(), u=u.data_ptr(), unit=unit.data_ptr())
    for c0 in range(0, plan.count, per_pass):
        p.c.c0, p.c.c1 = c0, min(plan.count, c0 + per_pass)
        N.call("sl_delta_chunks", C.byref(p), qo_indptr.numel() - 1, N.stream())
