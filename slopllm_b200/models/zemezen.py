"""Zemezen: a small decoder whose layers each name a mixer (grouped-query attention whose values are its key projections, latent
attention without positions, or a gated delta rule with a decay per key channel) and optionally a feed-forward (dense or routed
experts) that runs beside the mixer on the same normed input.  Layers may share another layer's weights.

This file is the configuration, the checkpoint's tensor names and the assembly of the shared parts: mixers and the parallel
block (`models/mixers.py`), decoder loop and engine hooks (`models/stack.py`), cache (`kv/hybrid.py`).
"""
from __future__ import annotations

import dataclasses
import functools
import json
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

from ..ops import get_ops
from ..ops.delta import DeltaShape, DeltaWeights
from ..ops.grouped import GroupedShape, GroupedWeights
from ..ops.latent import LatentShape, LatentWeights
from ..ops.rotary import rotary_table
from ..parallel.dist import Comm, ParallelContext
from .mixers import ChannelDelta, Experts, GroupedAttention, LatentAttention, ParallelBlock
from .stack import DecoderStack, Sublayer
from .weights import ExpertWeights, LinearWeight

MIXER_KEYS = {"attention": ("heads", "kv_heads", "dim", "scale", "rot"), "latent_attention": ("heads", "dim", "vdim", "kv_rank", "scale"),
              "channel_delta": ("heads", "kv_heads", "dim", "vdim", "conv")}


@dataclass
class ZemezenExperts:
    count: int
    top: int
    ff: int
    groups: int = 1
    keep: int = 1


@dataclass
class ZemezenLayer:
    type: str
    mixer: dict
    ff: int = 0                                    # width of a dense feed-forward (0: none)
    experts: Optional[ZemezenExperts] = None
    weights_of: Optional[int] = None               # layer whose tensors this one uses


@dataclass
class ZemezenConfig:
    hidden_size: int
    vocab_size: int
    rms_norm_eps: float
    layers: List[ZemezenLayer]
    eos_token_ids: List[int] = field(default_factory=list)
    model_type: str = "zemezen"
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
            if "kv_heads" in c and c["heads"] % c["kv_heads"]:
                raise ValueError(f"layer {i}: {c['heads']} heads do not share {c['kv_heads']} key heads evenly")
            if l.type == "attention":
                if c["rot"]["dims"] % 2 or c["rot"]["dims"] > c["dim"]:
                    raise ValueError(f"layer {i}: rot.dims must be even and at most dim")
                if c.get("vdim", c["dim"]) != c["dim"]:
                    raise ValueError(f"layer {i}: values are key projections, so vdim must equal dim")
            if l.experts is not None:
                e = l.experts
                if e.count % e.groups or not 1 <= e.keep <= e.groups or not 1 <= e.top <= e.keep * (e.count // e.groups):
                    raise ValueError(f"layer {i}: {e.top} of {e.count} experts cannot be chosen from {e.keep} of {e.groups} groups")
            if l.weights_of is not None:
                src = self.layers[self.source(i)]
                if (l.type, l.mixer, l.ff, l.experts) != (src.type, src.mixer, src.ff, src.experts):
                    raise ValueError(f"layer {i} differs from layer {l.weights_of}, whose weights it uses")

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def source(self, i: int) -> int:
        """The layer whose tensors layer i uses."""
        seen = set()
        while self.layers[i].weights_of is not None:
            seen.add(i)
            i = self.layers[i].weights_of
            if not 0 <= i < len(self.layers) or i in seen:
                raise ValueError(f"weights_of leads to no layer with tensors (at {i})")
        return i

    @classmethod
    def from_dict(cls, raw: dict) -> "ZemezenConfig":
        layers = []
        for i, l in enumerate(raw["layers"]):
            mlp, ff, experts = l.get("mlp"), 0, None
            if mlp is not None and mlp.get("kind") == "dense":
                ff = int(mlp["ff"])
            elif mlp is not None and mlp.get("kind") == "moe":
                r = mlp["router"]
                g = r.get("groups") or {}
                experts = ZemezenExperts(int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"]), int(g.get("count", 1)), int(g.get("keep", 1)))
            elif mlp is not None:
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            layers.append(ZemezenLayer(l["type"], dict(l["mixer"]), ff, experts, l.get("weights_of")))
        eos = raw.get("eos_token_id", [])
        return cls(hidden_size=raw["width"], vocab_size=raw["vocab"], rms_norm_eps=raw["norm"]["eps"], layers=layers,
                   eos_token_ids=list(eos) if isinstance(eos, (list, tuple)) else [eos])

    @classmethod
    def tiny(cls) -> "ZemezenConfig":
        attn = {"heads": 4, "kv_heads": 2, "dim": 32, "scale": 32 ** -0.5, "rot": {"base": 10000.0, "dims": 16}, "mask": {"size": 24, "keep_first": 4}}
        delta = {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 48, "conv": 4}
        latent = {"heads": 4, "dim": 32, "vdim": 32, "kv_rank": 48, "scale": 32 ** -0.5}
        return cls(hidden_size=128, vocab_size=512, rms_norm_eps=1e-6, layers=[
            ZemezenLayer("channel_delta", delta, 192), ZemezenLayer("attention", attn, 0, ZemezenExperts(8, 2, 64, 4, 2)),
            ZemezenLayer("latent_attention", latent, 192), ZemezenLayer("channel_delta", delta, 192, weights_of=0)])


@dataclass
class ZemezenWeights:
    embed: torch.Tensor
    blocks: List[ParallelBlock]
    norms: List[torch.Tensor]                      # fp32, in front of each block
    final_norm: torch.Tensor                       # fp32
    lm_head: LinearWeight
    vocab_offset: int = 0


def random_zemezen_tensors(cfg: ZemezenConfig, seed: int = 0, low_rank: int = 16, device="cpu") -> Dict[str, torch.Tensor]:
    """Random checkpoint tensors (bf16) of a configuration, under the checkpoint's names."""
    g = torch.Generator(device=device).manual_seed(seed)
    H = cfg.hidden_size
    t: Dict[str, torch.Tensor] = {}

    def mat(name, n, k, gain=1.0):
        t[name] = (torch.randn(n, k, generator=g, device=device) * gain * k ** -0.5).to(torch.bfloat16)

    def vec(name, n, spread, shift=0.0):
        t[name] = (torch.randn(n, generator=g, device=device) * spread + shift).to(torch.bfloat16)

    def feed_forward(p, ff):
        mat(p + "gate", ff, H), mat(p + "up", ff, H), mat(p + "down", H, ff)

    t["embed"] = torch.randn(cfg.vocab_size, H, generator=g, device=device).to(torch.bfloat16)
    for i, l in enumerate(cfg.layers):
        if l.weights_of is not None:
            continue
        p, c = f"l{i}.", l.mixer
        vec(p + "norm1", H, 0.1, 1.0)
        if l.ff:
            feed_forward(p + "mlp.", l.ff)
        if l.experts is not None:
            for e in range(l.experts.count):
                feed_forward(f"{p}mlp.e{e}.", l.experts.ff)
            mat(p + "mlp.router", l.experts.count, H)
        p, h, d = p + "mix.", c["heads"], c["dim"]
        dv, kv = c.get("vdim", d), c.get("kv_heads", h)
        mat(p + "o", H, h * dv)
        if l.type == "attention":
            mat(p + "q", h * d, H), mat(p + "k", kv * d, H)
            vec(p + "q.norm", d, 0.1, 1.0), vec(p + "k.norm", d, 0.1, 1.0), vec(p + "sink", h, 1.0)
        elif l.type == "latent_attention":
            mat(p + "q", h * d, H), mat(p + "dkv", c["kv_rank"], H), vec(p + "dkv.norm", c["kv_rank"], 0.1, 1.0)
            mat(p + "uk", h * d, c["kv_rank"]), mat(p + "uv", h * dv, c["kv_rank"])
        else:
            for n, rows in (("q", kv * d), ("k", kv * d), ("v", h * dv)):
                mat(p + n, rows, H), mat(p + n + ".conv", rows, c["conv"], 1.5)
            mat(p + "b", h, H), vec(p + "A_log", h, 0.5), vec(p + "norm", dv, 0.1, 1.0), vec(p + "dt_bias", h * d, 1.0, -3.0)
            mat(p + "a1", low_rank, H), mat(p + "a2", h * d, low_rank), mat(p + "g1", low_rank, H), mat(p + "g2", h * dv, low_rank)
    vec("final.norm", H, 0.1, 1.0)
    mat("head", cfg.vocab_size, H)
    return t


def assemble_zemezen_weights(cfg: ZemezenConfig, tensors: Dict[str, torch.Tensor], device, dtype, rank: int = 0,
                             world: int = 1) -> ZemezenWeights:
    """Checkpoint tensors -> fused, tensor-parallel runtime weights: a layer's input projections (mixer and feed-forward) are
    stacked into one matrix, its output projections stand side by side in another; heads, feed-forward rows and the experts' inner
    rows are sharded; norm weights, biases, decays, convolutions and sinks are kept in fp32."""
    H, eps = cfg.hidden_size, cfg.rms_norm_eps

    def get(name, *shape):
        if name not in tensors:
            raise KeyError(f"missing tensor {name}")
        t = tensors[name]
        if len(shape) != t.dim() or any(a is not None and a != b for a, b in zip(shape, t.shape)):
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
    cols = lambda t: share(t.t()).t()

    def mixer_parts(i, l):
        """(mixer, main rows, fine rows, output columns) of layer i, all this rank's."""
        m, c = f"l{i}.mix.", l.mixer
        h, d = c["heads"], c["dim"]
        kv, dv = c.get("kv_heads", h), c.get("vdim", d)
        if h % world or kv % world:
            raise ValueError(f"layer {i}: {h} heads and {kv} key heads cannot be shared by {world} ranks")
        hl, kl = h // world, kv // world
        o = cols(get(m + "o", H, h * dv))
        if l.type == "attention":
            mask = c.get("mask") or {}
            shape = GroupedShape(hl, kl, d, dv, float(c["scale"]), int(mask.get("size") or 0), int(mask.get("keep_first") or 0), eps, own_values=False)
            w = GroupedWeights(f32(get(m + "q.norm", d)), f32(get(m + "k.norm", d)), f32(share(get(m + "sink", h))))
            rot = rotary_table(c["rot"]["dims"], c["rot"]["base"]).to(device)
            return GroupedAttention(i, shape, rot, w), [heads(get(m + "q", h * d, H), h), heads(get(m + "k", kv * d, H), kv)], [], o
        if l.type == "latent_attention":
            R = c["kv_rank"]
            shape = LatentShape(hl, d, 0, dv, R, float(c["scale"]), 0, eps)
            uv = dev(heads(get(m + "uv", h * dv, R), h)).view(hl, dv, R)
            w = LatentWeights(norm=f32(get(m + "dkv.norm", R)), uk=dev(heads(get(m + "uk", h * d, R), h)).view(hl, d, R), uv=uv,
                              uv_t=uv.transpose(1, 2).contiguous())
            main = [heads(get(m + "q", h * d, H), h), get(m + "dkv", R, H)]
            return LatentAttention(i, shape, rotary_table(0, 1.0).to(device), None, w, None), main, [], o
        shape = DeltaShape(hl, kl, d, dv, int(c["conv"]), eps)
        rows = (("q", kv * d, kv), ("k", kv * d, kv), ("v", h * dv, h))
        main = [heads(get(m + n, r, H), u) for n, r, u in rows]
        conv = torch.cat([heads(get(m + n + ".conv", r, shape.taps), u) for n, r, u in rows], 0)
        a1, g1 = get(m + "a1", None, H), get(m + "g1", None, H)
        w = DeltaWeights(conv=f32(conv.t()), a2=dev(heads(get(m + "a2", h * d, a1.shape[0]), h)), g2=dev(heads(get(m + "g2", h * dv, g1.shape[0]), h)),
                         dt_bias=f32(heads(get(m + "dt_bias", h * d), h)), A_log=f32(share(get(m + "A_log", h))), norm=f32(get(m + "norm", dv)))
        return ChannelDelta(i, shape, w), main, [a1, g1, share(get(m + "b", h, H))], o

    def build(i, l):
        mixer, main, fine, o = mixer_parts(i, l)
        p, ff, experts, outs, nfine = f"l{i}.mlp.", 0, None, [o], sum(t.shape[0] for t in fine)
        nmain = sum(t.shape[0] for t in main)
        if l.ff:
            ff = l.ff // world
            main += [share(get(p + "gate", l.ff, H)), share(get(p + "up", l.ff, H))]
            outs.append(cols(get(p + "down", H, l.ff)))
        if l.experts is not None:
            e = l.experts
            fine.append(get(p + "router", e.count, H))
            names = [f"{p}e{j}." for j in range(e.count)]
            w13 = torch.stack([torch.cat([share(get(n + "gate", e.ff, H)), share(get(n + "up", e.ff, H))]) for n in names])
            experts = Experts(ExpertWeights(dev(w13), dev(torch.stack([cols(get(n + "down", H, e.ff)) for n in names]))), e.top, e.groups, e.keep)
        return ParallelBlock(i, l.type, mixer, LinearWeight(dev(torch.cat(main + fine))), LinearWeight(dev(torch.cat(outs, 1))), nmain, o.shape[1], ff,
                             nfine, experts)

    made: Dict[int, ParallelBlock] = {}
    norm: Dict[int, torch.Tensor] = {}
    blocks, norms = [], []
    for i, l in enumerate(cfg.layers):
        j = cfg.source(i)
        if j not in made:
            made[j], norm[j] = build(j, cfg.layers[j]), f32(get(f"l{j}.norm1", H))
        b = made[j]
        # a layer that uses another's weights keeps a cache of its own
        blocks.append(b if i == j else dataclasses.replace(b, index=i, mixer=dataclasses.replace(b.mixer, index=i)))
        norms.append(norm[j])
    head = get("head", cfg.vocab_size, H)
    return ZemezenWeights(embed=dev(get("embed", cfg.vocab_size, H)), blocks=blocks, norms=norms, final_norm=f32(get("final.norm", H)),
                          lm_head=LinearWeight(dev(share(head))), vocab_offset=rank * (cfg.vocab_size // world))


class ZemezenModel(DecoderStack):
    fp32_norms = True

    def __init__(self, cfg: ZemezenConfig, weights: ZemezenWeights, ctx: Optional[ParallelContext] = None, ops=None,
                 comm: Optional[Comm] = None):
        self.cfg, self.w = cfg, weights
        ctx = ctx or ParallelContext(device=weights.embed.device)
        dtype = weights.embed.dtype
        self.specs = [b.spec for b in weights.blocks]
        self.sublayers = [Sublayer(functools.partial(b, self), n) for b, n in zip(weights.blocks, weights.norms)]
        self._init_stack(ctx, ops or get_ops(cfg, ctx.device, ctx, dtype), comm, dtype)

    @classmethod
    def from_tensors(cls, cfg: ZemezenConfig, tensors: Dict[str, torch.Tensor], ctx: Optional[ParallelContext] = None,
                     dtype=torch.bfloat16) -> "ZemezenModel":
        ctx = ctx or ParallelContext()
        w = assemble_zemezen_weights(cfg, tensors, ctx.device, dtype, ctx.rank if ctx.world > 1 else 0, ctx.world)
        return cls(cfg, w, ctx)


def load_zemezen_model(model_dir: str, ctx: Optional[ParallelContext] = None, dtype=torch.bfloat16):
    """(cfg, model) from a directory of config.json and safetensors shards."""
    from ..checkpoint.safetensors_io import load_dir
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = ZemezenConfig.from_dict(json.load(f))
    return cfg, ZemezenModel.from_tensors(cfg, load_dir(model_dir), ctx, dtype)
