"""Pulunex: a small decoder whose layers read their input mixed with the previous token's, attend inside chunks of the sequence with
talking heads (every head's scores are a mixture of all heads'), some of them over an earlier layer's keys and values, and feed a dense
or a routed feed-forward (correction of the choice, identity experts, gated shared expert).  Positions enter through learned vectors;
a norm's weight is one number.

This file is the configuration, the checkpoint's tensor names and the assembly of the shared parts: mixers and feed-forwards
(`models/mixers.py`), decoder loop and engine hooks (`models/stack.py`), cache (`kv/hybrid.py`).
"""
from __future__ import annotations

import dataclasses
import functools
import json
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

from ..kv.hybrid import CacheSpec
from ..ops import get_ops
from ..ops.talking import TalkingShape, TalkingWeights
from ..parallel.dist import Comm, ParallelContext
from .mixers import Experts, FeedForward, RoutedFeedForward, TalkingAttention
from .stack import DecoderStack, Sublayer, TokenShift
from .weights import ExpertWeights, LinearWeight

MIXER_KEYS = {"attention": ("heads", "kv_heads", "dim", "vdim", "scale")}


@dataclass
class PulunexExperts:
    count: int                       # experts with weights
    top: int
    ff: int
    identity: int = 0                # router outputs behind them that hand the input through
    shared_ff: int = 0               # width of the shared expert (0: none)


@dataclass
class PulunexLayer:
    type: str
    mixer: dict
    ff: int = 0                      # width of a dense feed-forward (0: none)
    experts: Optional[PulunexExperts] = None

    @property
    def kv_from(self) -> Optional[int]:
        return self.mixer.get("kv_from")

    @property
    def chunk(self) -> int:
        return int((self.mixer.get("mask") or {}).get("size") or 0)


@dataclass
class PulunexConfig:
    hidden_size: int
    vocab_size: int
    rms_norm_eps: float
    max_positions: int               # rows of the position table: no sequence is longer
    layers: List[PulunexLayer]
    embed_scale: float = 1.0
    logit_scale: float = 1.0
    eos_token_ids: List[int] = field(default_factory=list)
    model_type: str = "pulunex"
    num_nextn_predict_layers: int = 0

    def __post_init__(self):
        if not self.layers:
            raise ValueError("the configuration lists no layers")
        for i, l in enumerate(self.layers):
            c = l.mixer
            if l.type not in MIXER_KEYS:
                raise ValueError(f"layer {i}: unknown mixer {l.type!r}")
            missing = [k for k in MIXER_KEYS[l.type] if k not in c]
            if missing:
                raise ValueError(f"layer {i} ({l.type}): missing {', '.join(missing)}")
            if c["heads"] % c["kv_heads"]:
                raise ValueError(f"layer {i}: {c['heads']} heads do not share {c['kv_heads']} key heads evenly")
            if l.chunk < 0:
                raise ValueError(f"layer {i}: mask.size must not be negative")
            if l.kv_from is not None:
                if not 0 <= l.kv_from < i or self.layers[l.kv_from].kv_from is not None:
                    raise ValueError(f"layer {i}: kv_from must name an earlier layer with keys of its own")
                src = self.layers[l.kv_from].mixer
                if any(c[k] != src[k] for k in ("kv_heads", "dim", "vdim")):
                    raise ValueError(f"layer {i} differs in its key heads from layer {l.kv_from}, whose keys it uses")
            if l.experts is not None and not 1 <= l.experts.top <= l.experts.count + l.experts.identity:
                raise ValueError(f"layer {i}: {l.experts.top} of {l.experts.count + l.experts.identity} experts cannot be chosen")

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, raw: dict) -> "PulunexConfig":
        layers = []
        for i, l in enumerate(raw["layers"]):
            mlp, ff, experts = l.get("mlp"), 0, None
            if mlp is not None and mlp.get("kind") == "dense":
                ff = int(mlp["ff"])
            elif mlp is not None and mlp.get("kind") == "moe":
                r, shared = mlp["router"], mlp.get("shared")
                experts = PulunexExperts(int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"]), int(r.get("identity") or 0),
                                         int(shared["ff"]) if shared else 0)
            elif mlp is not None:
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            layers.append(PulunexLayer(l["type"], dict(l["mixer"]), ff, experts))
        eos = raw.get("eos_token_id", [])
        return cls(hidden_size=raw["width"], vocab_size=raw["vocab"], rms_norm_eps=raw["norm"]["eps"], max_positions=int(raw["max_positions"]),
                   layers=layers, embed_scale=float(raw["embedding"]["scale"]), logit_scale=float(raw["logit_scale"]),
                   eos_token_ids=list(eos) if isinstance(eos, (list, tuple)) else [eos])

    @classmethod
    def tiny(cls) -> "PulunexConfig":
        c = {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 48, "scale": 0.2, "mask": {"size": 40}}
        return cls(hidden_size=128, vocab_size=512, rms_norm_eps=1e-6, max_positions=4096, embed_scale=0.7, logit_scale=0.8, layers=[
            PulunexLayer("attention", c, 192), PulunexLayer("attention", c, 0, PulunexExperts(6, 2, 64, 2, 96)),
            PulunexLayer("attention", {**c, "kv_from": 1, "mask": {"size": 100}}, 0, PulunexExperts(8, 3, 64))])


@dataclass
class PulunexWeights:
    embed: torch.Tensor
    positions: torch.Tensor          # [max_positions, H]: added to the scaled token vectors
    sublayers: List[Sublayer]        # `run` takes the model first
    mixers: List[TalkingAttention]
    final_norm: torch.Tensor         # fp32, with the factor on the logits
    lm_head: LinearWeight
    embed_scale: float = 1.0
    vocab_offset: int = 0


def random_pulunex_tensors(cfg: PulunexConfig, seed: int = 0, device="cpu") -> Dict[str, torch.Tensor]:
    """Random checkpoint tensors (bf16) of a configuration, under the checkpoint's names."""
    g = torch.Generator(device=device).manual_seed(seed)
    H = cfg.hidden_size
    t: Dict[str, torch.Tensor] = {}

    def put(name, *shape, k=1.0, shift=0.0):
        t[name] = (torch.randn(shape, generator=g, device=device) * k + shift).to(torch.bfloat16)

    def mat(name, n, k):
        put(name, n, k, k=k ** -0.5)

    def swiglu(p, ff):
        mat(p + "gate", ff, H), mat(p + "up", ff, H), mat(p + "down", H, ff)

    put("embed", cfg.vocab_size, H), put("pos", cfg.max_positions, H, k=0.3)
    for i, l in enumerate(cfg.layers):
        p, c = f"l{i}.", l.mixer
        put(p + "norm1", k=0.1, shift=1.0), put(p + "shift", H, k=0.2, shift=0.3)
        m = p + "mix."
        rows = [("q", c["heads"] * c["dim"])]
        if l.kv_from is None:
            rows += [("k", c["kv_heads"] * c["dim"]), ("v", c["kv_heads"] * c["vdim"])]
        for n, r in rows:
            mat(m + n, r, H), put(m + n + ".b", r, k=0.1)
        t[m + "talk"] = (torch.eye(c["heads"], device=device) + torch.randn(c["heads"], c["heads"], generator=g, device=device) * 0.2).to(torch.bfloat16)
        mat(m + "o", H, c["heads"] * c["vdim"])
        m = p + "mlp."
        if l.ff or l.experts is not None:
            put(p + "norm2", k=0.1, shift=1.0)
        if l.ff:
            mat(m + "up", l.ff, H), mat(m + "down", H, l.ff)
        if l.experts is not None:
            e = l.experts
            for j in range(e.count):
                swiglu(f"{m}e{j}.", e.ff)
            mat(m + "router", e.count + e.identity, H), put(m + "correction", e.count + e.identity, k=0.02)
            if e.shared_ff:
                swiglu(m + "shared.", e.shared_ff), mat(m + "shared.sg", 1, H)
    put("final.norm", k=0.1, shift=1.0), mat("head", cfg.vocab_size, H)
    return t


def assemble_pulunex_weights(cfg: PulunexConfig, tensors: Dict[str, torch.Tensor], device, dtype, rank: int = 0, world: int = 1) -> PulunexWeights:
    """Checkpoint tensors -> fused, tensor-parallel runtime weights: a layer's input projections are stacked into one matrix, the shared
    expert's with the router's; value heads with the query heads that read them, feed-forward rows and the experts' inner rows are
    sharded.  Mixed scores need every head's, so query and key projections are whole on every rank.  Norms (spread over the row), biases,
    mixtures and corrections are kept in fp32."""
    H, eps = cfg.hidden_size, cfg.rms_norm_eps

    def get(name, *shape):
        if name not in tensors:
            raise KeyError(f"missing tensor {name}")
        t = tensors[name]
        if tuple(t.shape) != shape:
            raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {shape}")
        return t

    def share(t):
        """This rank's part of the first dimension."""
        if t.shape[0] % world:
            raise ValueError(f"{t.shape[0]} rows cannot be shared by {world} ranks")
        n = t.shape[0] // world
        return t[rank * n:(rank + 1) * n]

    def heads(t, h):
        return share(t.reshape(h, -1)).reshape(-1, *t.shape[1:])

    dev = lambda t: t.to(dtype).to(device).contiguous()
    f32 = lambda t: t.to(torch.float32).to(device).contiguous()
    lin = lambda *parts: LinearWeight(dev(torch.cat(parts, 0) if len(parts) > 1 else parts[0]))
    cols = lambda t: share(t.t()).t()

    def row(name, factor=1.0):
        """A norm's one number, spread over the row."""
        return f32(get(name).to(torch.float32).expand(H) * factor)

    def attention(i, l):
        p, c = f"l{i}.mix.", l.mixer
        h, kv, d, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
        if h % world or kv % world:
            raise ValueError(f"layer {i}: {h} heads and {kv} key heads cannot be shared by {world} ranks")
        own = l.kv_from is None
        rows, bias = [get(p + "q", h * d, H)], [get(p + "q.b", h * d)]
        if own:
            rows += [get(p + "k", kv * d, H), heads(get(p + "v", kv * dv, H), kv)]
            bias += [get(p + "k.b", kv * d), heads(get(p + "v.b", kv * dv), kv)]
        shape = TalkingShape(h, kv, h // world, kv // world, d, dv, float(c["scale"]), l.chunk, eps, own)
        w = TalkingWeights(f32(torch.cat(bias)), f32(share(get(p + "talk", h, h))), torch.ones(d, dtype=torch.float32, device=device))
        return TalkingAttention(i, i if own else l.kv_from, shape, w, lin(*rows), LinearWeight(dev(cols(get(p + "o", H, h * dv)))))

    def routed(i, e):
        p = f"l{i}.mlp."
        names = [f"{p}e{j}." for j in range(e.count)]
        w13 = torch.stack([torch.cat([share(get(n + "gate", e.ff, H)), share(get(n + "up", e.ff, H))]) for n in names])
        w2 = torch.stack([cols(get(n + "down", H, e.ff)) for n in names])
        outputs = e.count + e.identity
        experts = Experts(ExpertWeights(dev(w13), dev(w2)), e.top, correction=f32(get(p + "correction", outputs)), identity=rank == 0)
        fine, main, down = [get(p + "router", outputs, H)], [], None
        if e.shared_ff:
            s = p + "shared."
            main = [share(get(s + "gate", e.shared_ff, H)), share(get(s + "up", e.shared_ff, H))]
            fine.append(get(s + "sg", 1, H))
            down = LinearWeight(dev(cols(get(s + "down", H, e.shared_ff))))
        return RoutedFeedForward(i, lin(*main, *fine), down, e.shared_ff // world, outputs, experts)

    subs: List[Sublayer] = []
    mixers = []
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        mixers.append(attention(i, l))
        subs.append(Sublayer(mixers[-1], row(p + "norm1"), shift=TokenShift(i, f32(get(p + "shift", H)))))
        if l.ff:
            subs.append(Sublayer(FeedForward(i, lin(share(get(p + "mlp.up", l.ff, H))), LinearWeight(dev(cols(get(p + "mlp.down", H, l.ff)))), "gelu_tanh"),
                                 row(p + "norm2")))
        if l.experts is not None:
            subs.append(Sublayer(routed(i, l.experts), row(p + "norm2")))
    head = get("head", cfg.vocab_size, H)
    return PulunexWeights(embed=dev(get("embed", cfg.vocab_size, H)), positions=dev(get("pos", cfg.max_positions, H)), sublayers=subs, mixers=mixers,
                          final_norm=row("final.norm", cfg.logit_scale), lm_head=LinearWeight(dev(share(head))), embed_scale=cfg.embed_scale,
                          vocab_offset=rank * (cfg.vocab_size // world))


class PulunexModel(DecoderStack):
    fp32_norms = True

    def __init__(self, cfg: PulunexConfig, weights: PulunexWeights, ctx: Optional[ParallelContext] = None, ops=None, comm: Optional[Comm] = None):
        self.cfg, self.w = cfg, weights
        ctx = ctx or ParallelContext(device=weights.embed.device)
        dtype = weights.embed.dtype
        self.specs = [CacheSpec(m.spec.rows, {**m.spec.state, "shift": (cfg.hidden_size,)}) for m in weights.mixers]
        self.sublayers = [dataclasses.replace(s, run=functools.partial(s.run, self)) for s in weights.sublayers]
        self._init_stack(ctx, ops or get_ops(cfg, ctx.device, ctx, dtype), comm, dtype)

    @classmethod
    def from_tensors(cls, cfg: PulunexConfig, tensors: Dict[str, torch.Tensor], ctx: Optional[ParallelContext] = None,
                     dtype=torch.bfloat16) -> "PulunexModel":
        ctx = ctx or ParallelContext()
        w = assemble_pulunex_weights(cfg, tensors, ctx.device, dtype, ctx.rank if ctx.world > 1 else 0, ctx.world)
        return cls(cfg, w, ctx)


def load_pulunex_model(model_dir: str, ctx: Optional[ParallelContext] = None, dtype=torch.bfloat16):
    """(cfg, model) from a directory of config.json and safetensors shards."""
    from ..checkpoint.safetensors_io import load_dir
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = PulunexConfig.from_dict(json.load(f))
    return cfg, PulunexModel.from_tensors(cfg, load_dir(model_dir), ctx, dtype)
