"""Token shift: a layer reads its normed input mixed with the previous token's, in the same pass that joins the residual and normalises.

    h_t   = rms(residual_t) * w
    out_t = h_t + (h_{t-1} - h_t) * mix

h of a sequence's last token is per-sequence state; a sequence's first token has zeros in front.  The first pass of a step makes the
residual from the embedding table instead, with a factor and learned position vectors.  CUDA tensors run `csrc/token_shift.cu`, CPU
tensors the fp32 definition below.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch

from . import reference as R


def _native():
    from . import native as N
    return N


class ShiftNormParams(C.Structure):
    _fields_ = [("out", C.c_void_p), ("out_f32", C.c_int), ("res_out", C.c_void_p), ("y", C.c_void_p), ("ldy", C.c_int), ("res_in", C.c_void_p),
                ("ids", C.c_void_p), ("table", C.c_void_p), ("table_f32", C.c_int), ("vocab", C.c_int), ("scale", C.c_float), ("places", C.c_void_p),
                ("num_places", C.c_int), ("w", C.c_void_p), ("mix", C.c_void_p), ("state", C.c_void_p), ("positions", C.c_void_p),
                ("batch_idx", C.c_void_p), ("qo", C.c_void_p), ("slots", C.c_void_p), ("H", C.c_int), ("eps", C.c_float), ("guard", C.c_void_p)]


@dataclass
class Shift:
    mix: torch.Tensor          # fp32 [H]
    state: torch.Tensor        # fp32 [slots, H]: h of each sequence's last token
    qo: torch.Tensor           # int32 [B + 1]: token range of every sequence of the step
    slots: torch.Tensor        # int32 [B]
    batch_idx: torch.Tensor    # int32 [T]

    def apply(self, h: torch.Tensor) -> torch.Tensor:
        """The definition; leaves the new state."""
        before = torch.empty_like(h)
        before[1:] = h[:-1]
        for b in range(self.qo.numel() - 1):
            lo, hi, slot = int(self.qo[b]), int(self.qo[b + 1]), int(self.slots[b])
            before[lo] = self.state[slot]
            self.state[slot] = h[hi - 1]
        return h + (before - h) * self.mix


def _run(T: int, H: int, w, eps: float, shift: Optional[Shift], dtype, dev, positions, **src):
    N = _native()
    from . import tcgen05
    out = torch.empty(T, H, dtype=dtype, device=dev)
    res = torch.empty(T, H, dtype=torch.float32, device=dev)
    if shift is not None:
        src.update(mix=shift.mix.data_ptr(), state=shift.state.data_ptr(), qo=shift.qo.data_ptr(), slots=shift.slots.data_ptr(),
                   batch_idx=shift.batch_idx.data_ptr())
    p = ShiftNormParams(out=out.data_ptr(), out_f32=int(dtype == torch.float32), res_out=res.data_ptr(), w=w.data_ptr(), positions=positions.data_ptr(), H=H, eps=float(eps),
                        guard=tcgen05.error_flag(dev).data_ptr() + 16, **src)
    N.call("sl_shift_norm", C.byref(p), T, N.stream())
    return out, res


def embed_shift_norm(st, table: torch.Tensor, scale: float, places: Optional[torch.Tensor], w: torch.Tensor, eps: float, shift: Optional[Shift], dtype):
    """residual = table[ids] * scale + places[positions]; returns (its norm, shifted if `shift`; residual).  `places` (learned position
    vectors, of the table's type) may be None."""
    if table.is_cuda:
        ids = st.input_ids.to(torch.int64).contiguous()
        return _run(ids.shape[0], table.shape[1], w, eps, shift, dtype, table.device, st.positions, ids=ids.data_ptr(), table=table.data_ptr(),
                    table_f32=int(table.dtype == torch.float32), vocab=table.shape[0], scale=scale,
                    places=0 if places is None else places.data_ptr(), num_places=0 if places is None else places.shape[0])
    r = table[st.input_ids.to(torch.int64)].to(torch.float32) * scale
    if places is not None:
        r = r + places[st.positions.to(torch.int64)].to(torch.float32)
    h = R.rmsnorm(r, w, eps)
    return (h if shift is None else shift.apply(h)), r


def add_shift_norm(st, y: torch.Tensor, residual: torch.Tensor, w: torch.Tensor, eps: float, shift: Optional[Shift], dtype):
    """residual' = residual + y; returns (its norm, shifted if `shift`; residual')."""
    if y.is_cuda:
        if y.dtype != torch.float32 or y.stride(-1) != 1:
            y = y.to(torch.float32).contiguous()
        return _run(*y.shape, w, eps, shift, dtype, y.device, st.positions, y=y.data_ptr(), ldy=y.stride(0), res_in=residual.data_ptr())
    r = residual + y
    h = R.rmsnorm(r, w, eps)
    return (h if shift is None else shift.apply(h)), r
