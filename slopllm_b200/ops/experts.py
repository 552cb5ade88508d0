"""Mixture of small SwiGLU experts with bf16 or fp32 weights: softmax routing limited to groups of neighbours, with an optional
correction of the choice, and the weighted sum of the chosen experts added to an output row.  Ids behind the experts' are identity
experts: their output is the input.

CUDA tensors run `csrc/moe_stream.cu` (routing; streaming kernels for few rows, fp32 and odd sizes) and the grouped tcgen05 GEMMs
of `ops/gemm.py` (many rows); CPU tensors run the fp32 definition below.
"""
from __future__ import annotations

import ctypes as C

import torch

from . import reference as R

STREAM_MAX_T = 32          # rows up to which an expert's weights are streamed past its tokens


def _native():
    from . import native as N
    return N


class ExpertStreamParams(C.Structure):
    _fields_ = [("x", C.c_void_p), ("ldx", C.c_int), ("ids", C.c_void_p), ("wts", C.c_void_p), ("T", C.c_int), ("top", C.c_int),
                ("H", C.c_int), ("I", C.c_int), ("E", C.c_int), ("w13", C.c_void_p), ("w2", C.c_void_p), ("act", C.c_void_p),
                ("y_route", C.c_void_p), ("out", C.c_void_p), ("ldo", C.c_int), ("identity", C.c_int)]


def route_softmax(logits: torch.Tensor, top: int, groups: int = 1, keep: int = 1, correction: torch.Tensor | None = None):
    """Scores are the softmax over all experts; experts are chosen by score + `correction` (fp32 [E]; None: by score).  Experts form
    `groups` equal runs of neighbours; only those of the `keep` groups with the largest single choice can be chosen.  Returns (ids int32
    [T, top], weights fp32 [T, top]): the `top` largest choices (ties: lower id) and their scores as they are."""
    T, E = logits.shape
    if logits.is_cuda:
        N = _native()
        ids = torch.empty(T, top, dtype=torch.int32, device=logits.device)
        wts = torch.empty(T, top, dtype=torch.float32, device=logits.device)
        N.call("sl_route_softmax", ids.data_ptr(), wts.data_ptr(), logits.data_ptr(), logits.stride(0), N.ptr(correction), T, E, top, groups, keep,
               N.stream())
        return ids, wts
    s = torch.softmax(logits.to(torch.float32), -1)
    c = s if correction is None else s + correction
    best = R._stable_topk(c.view(T, groups, -1).amax(-1), keep)
    kept = torch.zeros(T, groups, dtype=torch.bool).scatter_(1, best, True).repeat_interleave(E // groups, 1)
    ids = R._stable_topk(c.masked_fill(~kept, float("-inf")), top)
    return ids.to(torch.int32), s.gather(1, ids)


def add_experts(x: torch.Tensor, experts, ids: torch.Tensor, wts: torch.Tensor, out: torch.Tensor, ops, identity: bool = False) -> None:
    """out [T, H] (fp32) += sum of the chosen experts' outputs times their weights.  Ids from the number of experts on belong to identity
    experts, which are left out unless `identity`."""
    T, H = x.shape
    I, E = experts.inter, experts.num_experts
    if not x.is_cuda:
        real = ids < E
        out += R.moe_experts(x, experts, ids.masked_fill(~real, 0), wts * real)
        if identity:
            out += x.to(torch.float32) * (wts * ~real).sum(-1, keepdim=True)
        return
    N = _native()
    if x.dtype == torch.bfloat16 and T > STREAM_MAX_T and H % 8 == 0 and I % 8 == 0 and E < 1024 and out.is_contiguous():
        from .gemm import moe_large
        moe_large(ops, x, experts, None, ids, wts, out=out)
        if identity:
            N.call("sl_identity_experts", out.data_ptr(), out.stride(0), x.data_ptr(), x.stride(0), ids.data_ptr(), wts.data_ptr(), T, ids.shape[1], H, E,
                   int(x.dtype == torch.float32), N.stream())
        return
    k = ids.shape[1]
    act = torch.empty(T * k, I, dtype=x.dtype, device=x.device)
    y = torch.empty(T * k, H, dtype=torch.float32, device=x.device)
    p = ExpertStreamParams(x=x.data_ptr(), ldx=x.stride(0), ids=ids.data_ptr(), wts=wts.data_ptr(), T=T, top=k, H=H, I=I, E=E,
                           w13=experts.w13.data_ptr(), w2=experts.w2.data_ptr(), act=act.data_ptr(), y_route=y.data_ptr(),
                           out=out.data_ptr(), ldo=out.stride(0), identity=int(identity))
    N.call("sl_expert_stream", C.byref(p), int(x.dtype == torch.float32), N.stream())
