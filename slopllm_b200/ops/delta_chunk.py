"""Chunked form of the channel-wise gated delta rule (`csrc/delta_chunk.cu`): allocation, passes and launches."""
from __future__ import annotations

import ctypes as C

import torch

from .recurrent import CHUNK, CHUNK_MIN_Q, GatedScanParams

SCRATCH_BYTES = 256 << 20           # operands and states of the chunks of one pass; longer steps run in several passes


class DeltaChunkParams(C.Structure):
    _fields_ = [("s", GatedScanParams), ("chunks", C.c_void_p), ("seq_chunks", C.c_void_p), ("c0", C.c_int), ("c1", C.c_int), ("z", C.c_void_p),
                ("dt_bias", C.c_void_p), ("A_log", C.c_void_p), ("beta", C.c_void_p), ("ld_beta", C.c_int), ("unit_eps", C.c_float),
                ("w", C.c_void_p), ("kt", C.c_void_p), ("qt", C.c_void_p), ("pm", C.c_void_p), ("decay", C.c_void_p), ("u0", C.c_void_p),
                ("u", C.c_void_p), ("sin", C.c_void_p), ("stages", C.c_int)]


def scratch_parts(dk: int, dv: int) -> dict:
    """Bytes per (chunk, head) of what the three kernels hand on (multiples of 16)."""
    return {"w": CHUNK * dk * 4, "kt": CHUNK * dk * 4, "qt": CHUNK * dk * 4, "pm": CHUNK * CHUNK * 4, "decay": dk * 4, "u0": CHUNK * dv * 4,
            "u": CHUNK * dv * 4, "sin": dk * dv * 4}


def scratch_bytes(dk: int, dv: int) -> int:
    return sum(scratch_parts(dk, dv).values())


def usable(s, plan, x, out) -> bool:
    from . import native as N
    return bool(plan is not None and plan.longest >= CHUNK_MIN_Q and x.dtype == torch.bfloat16 and out.dtype == torch.bfloat16
                and x.stride(0) % 8 == 0 and s.kv_heads * s.dk % 8 == 0 and out.stride(0) % 2 == 0 and N.fn("sl_delta_chunk_ok")(s.dk, s.dv))


def run(x, fine, s, w, S, qo_indptr, state_idx, out, ops, plan) -> None:
    """x bf16 [T, q | k | v channels] behind the convolutions, fine fp32 [T, decay rank | gate rank | heads (beta)]."""
    from ..models.weights import LinearWeight
    ra, rg = w.a2.shape[1], w.g2.shape[1]
    low = fine[:, :ra + rg].to(torch.bfloat16)
    z = ops.linear(low[:, :ra], LinearWeight(w.a2), out_f32=True)
    gate = ops.linear(low[:, ra:], LinearWeight(w.g2))
    run_chunks(x, z, gate, fine[:, ra + rg:], s, w, S, qo_indptr, state_idx, out, plan)


def run_chunks(x, z, gate, beta, s, w, S, qo_indptr, state_idx, out, plan) -> None:
    """The recurrence itself: z fp32 [T, heads * dk] (decay input without bias), gate bf16 [T, heads * dv], beta fp32 [T, heads]."""
    from . import native as N
    from .delta import UNIT_EPS
    h, dk, dv, qk = s.heads, s.dk, s.dv, s.kv_heads * s.dk
    if z.stride(0) != h * dk:
        z = z.contiguous()
    per_pass = min(plan.count, max(1, SCRATCH_BYTES // (h * scratch_bytes(dk, dv))))
    off, at_byte = 0, {}
    for name, nbytes in scratch_parts(dk, dv).items():
        at_byte[name] = off
        off += per_pass * h * nbytes
    scratch = torch.empty(off, dtype=torch.uint8, device=x.device)
    at = lambda i: x.data_ptr() + 2 * i
    sp = GatedScanParams(out=out.data_ptr(), q=at(0), k=at(qk), v=at(2 * qk), g=gate.data_ptr(), ld=x.stride(0), norm_w=w.norm.data_ptr(),
                         eps=s.eps, S=S.data_ptr(), qo_indptr=qo_indptr.data_ptr(), state_idx=state_idx.data_ptr(), h=h, dk=dk, dv=dv,
                         ldg=gate.stride(0), ldo=out.stride(0), group=h // s.kv_heads)
    p = DeltaChunkParams(s=sp, chunks=plan.table.data_ptr(), seq_chunks=plan.seq_chunks.data_ptr(), z=z.data_ptr(), dt_bias=w.dt_bias.data_ptr(),
                         A_log=w.A_log.data_ptr(), beta=beta.data_ptr(), ld_beta=beta.stride(0), unit_eps=UNIT_EPS,
                         **{name: scratch.data_ptr() + o for name, o in at_byte.items()})
    for c0 in range(0, plan.count, per_pass):
        p.c0, p.c1 = c0, min(plan.count, c0 + per_pass)
        N.call("sl_delta_chunks", C.byref(p), qo_indptr.numel() - 1, N.stream())
