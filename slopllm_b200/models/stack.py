"""The decoder loop and the engine hooks shared by the model families whose layers are mixer + feed-forward sublayers over a
:class:`~slopllm_b200.kv.hybrid.HybridCache`: Qwen3 / Qwen3.5 (`models/dense.py`), Gidisun (`models/gidisun.py`), Zemezen
(`models/zemezen.py`), Vononex (`models/vononex.py`) and Pulunex (`models/pulunex.py`).

A family builds a flat list of :class:`Sublayer`; the loop runs  x -> run(norm(x)) -> [post norm] -> residual add -> next norm,
or, in families that normalise the sum,  x -> norm(alpha x + run(x) + bias),  with the residual in fp32, and completes the
tensor-parallel partial sums in between.  What a sublayer reads may be mixed with what it read for the previous token.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable, List, Optional

import torch

from ..kv.hybrid import CacheSpec, HybridCache, StateSlots
from ..ops import shift as SH
from ..parallel.dist import Comm, ParallelContext


@dataclass
class TokenShift:
    """The normed input h becomes h + (h of the previous token - h) * mix; the last token's h is the layer's state "shift"."""

    index: int                                 # layer
    mix: torch.Tensor                          # fp32 [H]


@dataclass
class Sublayer:
    run: Callable                              # (x, st, cache) -> this rank's partial sum [T, H]
    norm: Optional[torch.Tensor]               # weight of the RMS norm in front (None: `run` reads the residual itself)
    post_norm: Optional[torch.Tensor] = None   # fp32 weight of the RMS norm on the output (None: the output is added as it is),
                                               # with `alpha` on the sum
    alpha: Optional[float] = None              # factor on the residual of a sublayer whose sum is normalised
    bias: Optional[torch.Tensor] = None        # fp32 [H], added to the complete output (sums that are normalised)
    shift: Optional[TokenShift] = None         # mixes the normed input with the previous token's


def token_ranges(st):
    """(qo_indptr, longest range) of a step: token range of every sequence, or (None, 1) when every page-table row has one
    token (a decode step)."""
    q = st.extra.get("qo_indptr")
    if q is not None:
        return q, st.extra.get("max_q", st.num_tokens)
    T, B = st.num_tokens, st.page_table.shape[0]
    if T == B:
        return None, 1
    return torch.tensor([0, T], dtype=torch.int32, device=st.input_ids.device), T


class DecoderStack:
    """Base of the mixer / feed-forward families.  Subclasses set `cfg`, `w` (with `embed`, `lm_head`, `final_norm`,
    `vocab_offset`), `sublayers` and `specs` before calling `_init_stack`."""

    sublayers: List[Sublayer]
    specs: List[CacheSpec]
    fp32_norms = False        # norm weights are fp32 although no sublayer has a post norm

    def _init_stack(self, ctx: ParallelContext, ops, comm: Optional[Comm], cache_dtype) -> None:
        self.ctx, self.ops, self.comm = ctx, ops, comm or Comm(ctx)
        self.cache_dtype = cache_dtype
        # a recurrent state needs one slot per live sequence, and prefix sharing cannot restore it
        self.supports_prefix_sharing = not any(s.state for s in self.specs)
        self.states: Optional[StateSlots] = None

    # ---- engine hooks ---------------------------------------------------------------------------------------------
    def _make_cache(self, num_pages: int, max_states: int) -> HybridCache:
        return HybridCache(self.specs, num_pages, self.ctx.device, max_states, self.cache_dtype)

    def allocate_cache(self, num_pages: int, max_states: int = 64) -> HybridCache:
        cache = self._make_cache(num_pages, max_states)
        self.states = None if self.supports_prefix_sharing else StateSlots(max_states, self.ctx.device, cache.reset_state)
        return cache

    def prepare_step(self, st, seqs) -> None:
        """Host-side, outside any graph capture: state slots of the step's sequences (zeroed on first use)."""
        if self.states is not None:
            self.states.assign([s.seq_id for s in seqs])

    def release_sequence(self, seq_id: int) -> None:
        if self.states is not None:
            self.states.release(seq_id)

    # ---- forward --------------------------------------------------------------------------------------------------
    def scan_ranges(self, st):
        """(qo_indptr, state slot of each range) for the recurrent kernels."""
        qo, _ = token_ranges(st)
        if qo is None:
            qo = torch.arange(st.num_tokens + 1, dtype=torch.int32, device=st.input_ids.device)
        sidx = self.states.index if self.states is not None else torch.zeros(qo.numel() - 1, dtype=torch.int32, device=qo.device)
        return qo, sidx

    def _shift(self, shift: Optional[TokenShift], st, cache):
        if shift is None:
            return None
        return SH.Shift(shift.mix, cache.state[shift.index]["shift"], *self.scan_ranges(st), st.batch_idx)

    def _enter(self, st, cache, sub: Sublayer):
        ops, eps = self.ops, self.cfg.rms_norm_eps
        norm, places = sub.norm, getattr(self.w, "positions", None)
        if sub.shift is not None or places is not None:
            return SH.embed_shift_norm(st, self.w.embed, getattr(self.w, "embed_scale", 1.0), places, norm, eps, self._shift(sub.shift, st, cache),
                                       ops.act_dtype)
        if norm is None:
            return ops.embed_rows(st.input_ids, self.w.embed)
        if self.fp32_norms or self.sublayers[0].post_norm is not None:
            return ops.embed_norm(st.input_ids, self.w.embed, norm, eps)
        return ops.add_rmsnorm(ops.embed(st.input_ids, self.w.embed), None, norm, eps)

    def _join(self, y, residual, sub: Sublayer, nxt: Optional[Sublayer], st, cache):
        """`nxt`: the sublayer that reads the sum (None: the output head)."""
        ops, eps = self.ops, self.cfg.rms_norm_eps
        norm = self.w.final_norm if nxt is None else nxt.norm
        if nxt is not None and nxt.shift is not None:
            return SH.add_shift_norm(st, self.comm.all_reduce(y), residual, norm, eps, self._shift(nxt.shift, st, cache), ops.act_dtype)
        if sub.alpha is not None:
            return ops.sum_norm(self.comm.all_reduce(y), residual, sub.alpha, sub.bias, sub.post_norm, norm, eps)
        if self.fp32_norms or sub.post_norm is not None:
            return ops.post_norm(self.comm.all_reduce(y), residual, sub.post_norm, norm, eps)
        return self.comm.allreduce_add_rmsnorm(ops, y, residual, norm, eps)

    def forward_hidden(self, st, cache) -> torch.Tensor:
        x, residual = self._enter(st, cache, self.sublayers[0])
        for sub, nxt in zip(self.sublayers, [*self.sublayers[1:], None]):
            y = sub.run(x, st, cache)
            x, residual = self._join(y, residual, sub, nxt, st, cache)
        return x

    def compute_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        local = self.ops.logits(hidden, self.w.lm_head)
        if self.ctx.world == 1:
            return local
        return self.comm.all_gather(local, dim=-1)
