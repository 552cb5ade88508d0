"""Token mixers as building blocks: a mixer holds one layer's weights, says what it caches (:class:`CacheSpec`) and maps the
normed input [T, H] to this rank's partial output [T, H] (heads are sharded over the tensor-parallel ranks, the output
projection completes in the caller's all-reduce).  Every size and constant is a parameter, so any family can use them.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Union

import torch

from ..kv.hybrid import CacheSpec
from ..ops import delta as DL
from ..ops import experts as EX
from ..ops import grouped as G
from ..ops import latent as L
from ..ops import recurrent as RC
from ..ops import talking as TK
from ..ops.rotary import RotaryTable, Turn
from ..utils.tracing import traced
from .weights import ExpertWeights, LinearWeight

TOGETHER_MAX = 12 << 20      # output values of a step (tokens x width) up to which mixers side by side run at the same time: larger
                             # ones fill the GPU alone and only get in each other's way
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

    fp32_rows = False                # `mix` takes the projection in the activation type only

    def mix(self, model, qd, fine, st, cache, out=None):
        """Up to the output projection, from the rows of `w_in`."""
        rows = cache.rows[self.index]["latent"]
        q_rot = L.latent_pre(qd, self.shape, self.w, self.rot, st, rows)
        return L.latent_attention(qd, q_rot, self.shape, self.w, st, rows, model.ops, out)

    @traced(lambda self, *a, **k: f"layer{self.index}.latent_attention")
    def __call__(self, model, x, st, cache):
        return model.ops.linear(self.mix(model, model.ops.linear(x, self.w_in), None, st, cache), self.o_proj, out_f32=True)


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


@dataclass
class GroupedAttention:
    """Grouped-query attention with query / key norm, rotation, sliding window with kept first tokens and sink
    (`ops/grouped.py`).  Projection rows: q | k (| v)."""

    index: int
    shape: G.GroupedShape
    rot: RotaryTable
    w: G.GroupedWeights

    fp32_rows = True

    @property
    def spec(self) -> CacheSpec:
        s = self.shape
        return CacheSpec(rows={"k": (s.kv_heads, s.dim), "v": (s.kv_heads, s.vdim)})

    def mix(self, model, main, fine, st, cache, out):
        rows = cache.rows[self.index]
        q = G.grouped_pre(main, self.shape, self.w, self.rot, st, rows["k"], rows["v"], out.dtype)
        G.grouped_attention(q, self.shape, self.w, st, rows["k"], rows["v"], out)


@dataclass
class RowNormAttention:
    """Grouped-query attention with one norm over all heads' queries (and keys), biases, a factor per head on the scores and values
    that turn with their position (`ops/grouped.py`).  Projection rows: q | k | v, each head's in adjacent order."""

    index: int
    shape: G.GroupedShape
    turn: Turn
    v_turn: Optional[Turn]
    w: G.RowNormWeights
    scale: float = 1.0               # on the output

    @property
    def spec(self) -> CacheSpec:
        s = self.shape
        return CacheSpec(rows={"k": (s.kv_heads, s.dim), "v": (s.kv_heads, s.vdim)})

    def mix(self, model, main, fine, st, cache, out):
        rows, angles = cache.rows[self.index], model.angles.of(st)
        q = G.grouped_row_pre(main, self.shape, self.w, self.turn, self.v_turn, angles, st, rows["k"], rows["v"], out.dtype, model.comm)
        G.grouped_attention(q, self.shape, self.w, st, rows["k"], rows["v"], out, G.Finish(self.v_turn, angles, self.scale))


@dataclass
class Retention:
    """Linear attention with a fixed decay per head and rotated queries and keys (`ops/recurrent.py: retention_mix`).  Projection
    rows: q | k (each head's in adjacent order) | v | output gate."""

    index: int
    heads: int
    dk: int
    dv: int
    eps: float
    turn: Turn
    decay: torch.Tensor              # fp32 [2, heads], `recurrent.retention_decays`
    scale: float = 1.0               # on the output

    @property
    def spec(self) -> CacheSpec:
        return CacheSpec(state={"S": (self.heads, self.dk, self.dv)})

    def mix(self, model, main, fine, st, cache, out):
        qo, sidx = model.scan_ranges(st)
        RC.retention_mix(main, self.decay, self.turn, model.angles.of(st), self.eps, cache.state[self.index]["S"], qo, sidx, self.heads, self.dk,
                         self.dv, out, self.scale, RC.ChunkPlan.of(st))


@dataclass
class SideBySide:
    """Two mixers that read the same input and whose outputs are added: one input product makes the rows of both, which then run at
    the same time, and one output product takes their results side by side."""

    index: int
    kind: str
    parts: list                      # the mixers (with `mix`)
    rows: List[int]                  # projection rows of each
    outs: List[int]                  # values that each hands to `w_out`
    w_in: LinearWeight
    w_out: LinearWeight

    @property
    def spec(self) -> CacheSpec:
        return CacheSpec(rows={n: x for m in self.parts for n, x in m.spec.rows.items()},
                         state={n: x for m in self.parts for n, x in m.spec.state.items()})

    @traced(lambda self, *a, **k: f"layer{self.index}.{self.kind}")
    def __call__(self, model, x, st, cache):
        main = model.ops.linear(x, self.w_in, out_f32=x.shape[0] <= SMALL_T)
        both = torch.empty(x.shape[0], sum(self.outs), dtype=x.dtype, device=x.device)
        model.angles.of(st), RC.ChunkPlan.of(st)          # (made in front of the fork: both mixers read them)
        (a, b), r, o = self.parts, self.rows[0], self.outs[0]
        first = lambda: a.mix(model, main[:, :r], None, st, cache, both[:, :o])
        second = lambda: b.mix(model, main[:, r:r + self.rows[1]], None, st, cache, both[:, o:])
        if both.numel() <= TOGETHER_MAX:
            model.ops.together(first, second)
        else:
            first(), second()
        return model.ops.linear(both, self.w_out, out_f32=True)


@dataclass
class MinGru:
    """Element-wise gated recurrence with an output gate (`ops/recurrent.py: min_gru_mix`)."""

    index: int
    width: int
    w_in: LinearWeight               # z | candidate | output gate
    bias: torch.Tensor               # fp32 [z | candidate]
    o_proj: LinearWeight

    @property
    def spec(self) -> CacheSpec:
        return CacheSpec(state={"S": (self.width,)})

    @traced(lambda self, *a, **k: f"layer{self.index}.mingru")
    def __call__(self, model, x, st, cache):
        proj = model.ops.linear(x, self.w_in, out_f32=x.shape[0] <= SMALL_T)
        qo, sidx = model.scan_ranges(st)
        y = RC.min_gru_mix(proj, self.bias, cache.state[self.index]["S"], qo, sidx, self.width, x.dtype, RC.ChunkPlan.of(st))
        return model.ops.linear(y, self.o_proj, out_f32=True)


@dataclass
class GatedFeedForward:
    """act(gate x + b) * (up x + b'), projected down; the down projection's bias belongs to the caller's join."""

    index: int
    w_in: LinearWeight               # gate | up
    bias: Optional[torch.Tensor]     # fp32 [gate | up]
    w_out: LinearWeight
    act: str = "silu"

    @traced(lambda self, *a, **k: f"layer{self.index}.mlp")
    def __call__(self, model, x, st, cache):
        gu = model.ops.linear(x, self.w_in)
        act = torch.empty(x.shape[0], gu.shape[1] // 2, dtype=x.dtype, device=x.device)
        model.ops.gated_act(gu, act, self.act, self.bias)
        return model.ops.linear(act, self.w_out, out_f32=True)


@dataclass
class FeedForward:
    """act(up x), projected down."""

    index: int
    w_in: LinearWeight               # up
    w_out: LinearWeight
    act: str = "gelu_tanh"

    @traced(lambda self, *a, **k: f"layer{self.index}.mlp")
    def __call__(self, model, x, st, cache):
        up = model.ops.linear(x, self.w_in)
        act = torch.empty(x.shape[0], up.shape[1], dtype=x.dtype, device=x.device)
        model.ops.plain_act(up, act, self.act)
        return model.ops.linear(act, self.w_out, out_f32=True)


@dataclass
class TalkingAttention:
    """Grouped-query attention inside chunks whose heads' scores are mixed before the softmax, over its own keys and values or those of
    another layer's cache (`ops/talking.py`)."""

    index: int
    kv_index: int                    # layer whose cache holds the keys and values
    shape: TK.TalkingShape
    w: TK.TalkingWeights
    w_in: LinearWeight               # q (| k | v, with keys of its own)
    o_proj: LinearWeight

    @property
    def spec(self) -> CacheSpec:
        s = self.shape
        return CacheSpec(rows={"k": (s.kv_heads, s.dim), "v": (s.v_heads, s.vdim)}) if self.kv_index == self.index else CacheSpec()

    @traced(lambda self, *a, **k: f"layer{self.index}.talking_attention")
    def __call__(self, model, x, st, cache):
        s, rows = self.shape, cache.rows[self.kv_index]
        proj = model.ops.linear(x, self.w_in, out_f32=x.shape[0] <= SMALL_T)
        q = TK.talking_pre(proj, s, self.w, st, rows["k"], rows["v"], x.dtype)
        out = torch.empty(x.shape[0], s.out_heads * s.vdim, dtype=x.dtype, device=x.device)
        TK.talking_attention(q, s, self.w, st, rows["k"], rows["v"], out)
        return model.ops.linear(out, self.o_proj, out_f32=True)


@dataclass
class ChannelDelta:
    """Gated delta rule with a decay per key channel behind short convolutions (`ops/delta.py`).  Projection rows: q | k | v, and
    with fp32 results low-rank decay input | low-rank gate input | beta."""

    index: int
    shape: DL.DeltaShape
    w: DL.DeltaWeights

    fp32_rows = True

    @property
    def spec(self) -> CacheSpec:
        s = self.shape
        return CacheSpec(state={"S": (s.heads, s.dk, s.dv), "conv": (s.taps, s.channels)})

    def mix(self, model, main, fine, st, cache, out):
        state = cache.state[self.index]
        qo, sidx = model.scan_ranges(st)
        DL.channel_delta_mix(main, fine, self.shape, self.w, state["S"], state["conv"], st, qo, sidx, out, model.ops, RC.ChunkPlan.of(st))


@dataclass
class Experts:
    """Softmax-routed SwiGLU experts (`ops/experts.py`); the router's logits come from the caller's projection.  Router outputs behind the
    experts' are identity experts, whose output is the input."""

    w: ExpertWeights
    top: int
    groups: int = 1
    keep: int = 1
    correction: Optional[torch.Tensor] = None     # fp32, added to the scores when experts are chosen
    identity: bool = True                         # this rank adds the identity experts' outputs

    def add(self, model, x, logits, out):
        ids, wts = EX.route_softmax(logits, self.top, self.groups, self.keep, self.correction)
        EX.add_experts(x, self.w, ids, wts, out, model.ops, self.identity and logits.shape[1] > self.w.num_experts)


@dataclass
class RoutedFeedForward:
    """Routed experts and, if `w_out` is given, a shared expert behind a sigmoid gate: one product makes its rows, the router's logits and
    the gate."""

    index: int
    w_in: LinearWeight               # shared gate | shared up and then, with fp32 results, router | gate of the shared expert
    w_out: Optional[LinearWeight]
    ff: int                          # width of the shared expert
    outputs: int                     # of the router
    experts: Experts

    @traced(lambda self, *a, **k: f"layer{self.index}.moe")
    def __call__(self, model, x, st, cache):
        ops, T, m, w = model.ops, x.shape[0], 2 * self.ff, self.w_in.weight
        if w.dtype == torch.float32 or T <= SMALL_T:
            y = ops.linear(x, self.w_in, out_f32=True)
            main, fine = y[:, :m], y[:, m:]
        else:
            main, fine = ops.linear(x, LinearWeight(w[:m])) if m else None, ops.linear(x, LinearWeight(w[m:]), out_f32=True)
        if self.w_out is None:
            out = torch.zeros(T, x.shape[1], dtype=torch.float32, device=x.device)
        else:
            act = torch.empty(T, self.ff, dtype=x.dtype, device=x.device)
            ops.gated_act(main, act, "silu", row_gate=fine[:, self.outputs])
            out = ops.linear(act, self.w_out, out_f32=True)
        self.experts.add(model, x, fine[:, :self.outputs], out)
        return out


@dataclass
class ParallelBlock:
    """A mixer and a feed-forward that read the same normed input and whose outputs are added: one input product makes the rows of
    both, one output product takes the mixer's result and the activation side by side; routed experts add to its result.

    `w_in` rows: mixer | gate | up (dense feed-forward) and then, with fp32 results, the mixer's fine rows | router."""

    index: int
    kind: str
    mixer: Union[LatentAttention, GroupedAttention, ChannelDelta]
    w_in: LinearWeight
    w_out: LinearWeight
    main: int                        # mixer rows
    out: int                         # values the mixer hands to `w_out`
    ff: int = 0                      # width of the dense feed-forward
    fine: int = 0                    # the mixer's fine rows
    experts: Optional[Experts] = None

    @property
    def spec(self) -> CacheSpec:
        return self.mixer.spec

    @traced(lambda self, *a, **k: f"layer{self.index}.{self.kind}")
    def __call__(self, model, x, st, cache):
        ops, T, m, w = model.ops, x.shape[0], self.main + 2 * self.ff, self.w_in.weight
        if w.shape[0] == m:
            main, fine = ops.linear(x, self.w_in), None
        elif w.dtype == torch.float32 or (T <= SMALL_T and self.mixer.fp32_rows):
            y = ops.linear(x, self.w_in, out_f32=True)
            main, fine = y[:, :m], y[:, m:]
        else:
            main, fine = ops.linear(x, LinearWeight(w[:m])), ops.linear(x, LinearWeight(w[m:]), out_f32=True)
        both = torch.empty(T, self.out + self.ff, dtype=x.dtype, device=x.device)
        self.mixer.mix(model, main[:, :self.main], fine, st, cache, both[:, :self.out])
        if self.ff:
            ops.silu_mul(main[:, self.main:], both[:, self.out:])
        y = ops.linear(both, self.w_out, out_f32=True)
        if self.experts is not None:
            self.experts.add(model, x, fine[:, self.fine:], y)
        return y
