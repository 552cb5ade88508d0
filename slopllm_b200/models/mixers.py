"""Token mixers as building blocks: a mixer holds one layer's weights, says what it caches (:class:`CacheSpec`) and maps the
normed input [T, H] to this rank's partial output [T, H] (heads are sharded over the tensor-parallel ranks, the output
projection completes in the caller's all-reduce).  Every size and constant is a parameter, so any family can use them.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from ..kv.hybrid import CacheSpec
from ..ops import latent as L
from ..ops import recurrent as RC
from ..ops.rotary import RotaryTable
from ..utils.tracing import traced
from .weights import LinearWeight

SMALL_T = 32         # up to this many rows a layer's input projections are one fp32-output product (weight streaming)


@dataclass
class LatentAttention:
    """Latent attention with a shared rotated key part, sliding window and softmax sink (`ops/latent.py`)."""

    index: int
    shape: L.LatentShape
    rot: RotaryTable
    w_in: LinearWeight               # heads x (dim | rot_dim) query rows, rank latent rows, rot_dim shared key rows
    w: L.LatentWeights
    o_proj: LinearWeight

    @property
    def spec(self) -> CacheSpec:
        return CacheSpec(rows={"latent": (self.shape.row,)})

    @traced(lambda self, *a, **k: f"layer{self.index}.latent_attention")
    def __call__(self, model, x, st, cache):
        rows = cache.rows[self.index]["latent"]
        qd = model.ops.linear(x, self.w_in)
        q_rot = L.latent_pre(qd, self.shape, self.w, self.rot, st, rows)
        o = L.latent_attention(qd, q_rot, self.shape, self.w, st, rows, model.ops)
        return model.ops.linear(o, self.o_proj, out_f32=True)


class _GatedRecurrence:
    """Shared by the gated outer-product recurrences: `w_in` stacks q | k | v | output gate rows and then the rows that feed the
    gates of the recurrence, whose results stay fp32."""

    def _project(self, ops, x):
        main = self.heads * 2 * (self.dk + self.dv)
        if x.shape[0] <= SMALL_T:
            y = ops.linear(x, self.w_in, out_f32=True)
            return y, y[:, main:]
        w = self.w_in.weight
        return ops.linear(x, LinearWeight(w[:main])), ops.linear(x, LinearWeight(w[main:]), out_f32=True)


@dataclass
class GatedLinearAttention(_GatedRecurrence):
    """GLA: linear attention with a decay per key channel from a low-rank projection (`ops/recurrent.py: gla_mix`)."""

    index: int
    heads: int
    dk: int
    dv: int
    tau: float
    eps: float
    w_in: LinearWeight               # q | k | v | output gate | low-rank decay input
    a2: torch.Tensor                 # [heads * dk, rank]
    a2_b: torch.Tensor               # fp32 [heads * dk]
    norm: torch.Tensor               # fp32 [dv]
    o_proj: LinearWeight

    @property
    def spec(self) -> CacheSpec:
        return CacheSpec(state={"S": (self.heads, self.dk, self.dv)})

    @traced(lambda self, *a, **k: f"layer{self.index}.gla")
    def __call__(self, model, x, st, cache):
        proj, low = self._project(model.ops, x)
        qo, sidx = model.scan_ranges(st)
        o = RC.gla_mix(proj, low, self.a2, self.a2_b, self.tau, self.norm, self.eps, cache.state[self.index]["S"], qo, sidx,
                       self.heads, self.dk, self.dv, x.dtype, RC.ChunkPlan.of(st))
        return model.ops.linear(o, self.o_proj, out_f32=True)


@dataclass
class MLstm(_GatedRecurrence):
    """mLSTM: exponentially gated matrix memory with a normaliser state (`ops/recurrent.py: mlstm_mix`)."""

    index: int
    heads: int
    dk: int
    dv: int
    cap: float
    eps: float
    w_in: LinearWeight               # q | k | v | output gate | input gate | forget gate
    i_b: torch.Tensor                # fp32 [heads]
    f_b: torch.Tensor
    norm: torch.Tensor               # fp32 [heads * dv]
    o_proj: LinearWeight

    @property
    def spec(self) -> CacheSpec:
        return CacheSpec(state={"S": (self.heads, self.dk, self.dv), "n": (self.heads, self.dk), "m": (self.heads,)})

    @traced(lambda self, *a, **k: f"layer{self.index}.mlstm")
    def __call__(self, model, x, st, cache):
        proj, gates = self._project(model.ops, x)
        qo, sidx = model.scan_ranges(st)
        s = cache.state[self.index]
        o = RC.mlstm_mix(proj, gates, self.i_b, self.f_b, self.cap, self.norm, self.eps, (s["S"], s["n"], s["m"]), qo, sidx,
                         self.heads, self.dk, self.dv, x.dtype, RC.ChunkPlan.of(st))
        return model.ops.linear(o, self.o_proj, out_f32=True)
