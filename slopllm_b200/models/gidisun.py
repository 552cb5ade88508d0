"""Gidisun: a small decoder whose layers each name a mixer (latent attention with a sliding window and a sink, GLA or mLSTM)
and optionally a feed-forward, with a norm before and after every sublayer.

This file is the configuration, the checkpoint's tensor names and the assembly of the shared parts: mixers
(`models/mixers.py`), decoder loop and engine hooks (`models/stack.py`), cache (`kv/hybrid.py`).
"""
from __future__ import annotations

import functools
import json
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

from ..ops import get_ops
from ..ops.latent import LatentShape, LatentWeights
from ..ops.rotary import YarnScaling, rotary_table
from ..parallel.dist import Comm, ParallelContext
from ..utils.tracing import traced
from .mixers import GatedLinearAttention, LatentAttention, MLstm
from .stack import DecoderStack, Sublayer
from .weights import LinearWeight

MIXER_KEYS = {"latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot"),
              "gla": ("heads", "dim", "vdim", "tau"), "mlstm": ("heads", "dim", "vdim", "gate_cap")}


@dataclass
class GidisunLayer:
    type: str
    mixer: dict
    ff: int = 0                      # feed-forward width; 0: the layer has none


@dataclass
class GidisunConfig:
    hidden_size: int
    vocab_size: int
    rms_norm_eps: float
    layers: List[GidisunLayer]
    eos_token_ids: List[int] = field(default_factory=list)
    model_type: str = "gidisun"
    num_nextn_predict_layers: int = 0

    def __post_init__(self):
        for i, l in enumerate(self.layers):
            if l.type not in MIXER_KEYS:
                raise ValueError(f"layer {i}: unknown mixer {l.type!r}")
            missing = [k for k in MIXER_KEYS[l.type] if k not in l.mixer]
            if missing:
                raise ValueError(f"layer {i} ({l.type}): missing {', '.join(missing)}")
            if l.type == "latent_attention" and (l.mixer["rot"]["dims"] % 2 or l.mixer["rot"]["dims"] > l.mixer["rot_dim"]):
                raise ValueError(f"layer {i}: rot.dims must be even and at most rot_dim")
        if not self.layers:
            raise ValueError("the configuration lists no layers")

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, raw: dict) -> "GidisunConfig":
        layers = []
        for i, l in enumerate(raw["layers"]):
            mlp = l.get("mlp")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            layers.append(GidisunLayer(l["type"], dict(l["mixer"]), int(mlp["ff"]) if mlp else 0))
        eos = raw.get("eos_token_id", [])
        return cls(hidden_size=raw["width"], vocab_size=raw["vocab"], rms_norm_eps=raw["norm"]["eps"], layers=layers,
                   eos_token_ids=list(eos) if isinstance(eos, (list, tuple)) else [eos])

    @classmethod
    def tiny(cls) -> "GidisunConfig":
        attn = {"heads": 4, "dim": 32, "rot_dim": 16, "vdim": 32, "kv_rank": 48, "scale": 48 ** -0.5, "mask": {"size": 24},
                "rot": {"base": 10000.0, "dims": 16, "scaling": {"factor": 4.0, "original": 256, "fast": 32.0, "slow": 1.0}}}
        return cls(hidden_size=128, vocab_size=512, rms_norm_eps=1e-6, layers=[
            GidisunLayer("gla", {"heads": 4, "dim": 32, "vdim": 64, "tau": 16.0}, 192), GidisunLayer("latent_attention", attn, 192),
            GidisunLayer("mlstm", {"heads": 4, "dim": 48, "vdim": 32, "gate_cap": 15.0})])


@dataclass
class GidisunWeights:
    embed: torch.Tensor
    sublayers: List[Sublayer]        # `run` takes the model first
    mixers: list
    final_norm: torch.Tensor         # fp32
    lm_head: LinearWeight
    vocab_offset: int = 0


@dataclass
class DenseFeedForward:
    index: int
    mlp_w13: LinearWeight            # gate | up
    mlp_w2: LinearWeight

    @traced(lambda self, *a, **k: f"layer{self.index}.mlp")
    def __call__(self, model, x, st, cache):
        return model.ops.dense_mlp(x, self)


def random_gidisun_tensors(cfg: GidisunConfig, seed: int = 0, low_rank: int = 16, device="cpu") -> Dict[str, torch.Tensor]:
    """Random checkpoint tensors (bf16) of a configuration, under the checkpoint's names."""
    g = torch.Generator(device=device).manual_seed(seed)
    H = cfg.hidden_size
    t: Dict[str, torch.Tensor] = {}

    def mat(name, n, k):
        t[name] = (torch.randn(n, k, generator=g, device=device) * k ** -0.5).to(torch.bfloat16)

    def vec(name, n, spread, shift=0.0):
        t[name] = (torch.randn(n, generator=g, device=device) * spread + shift).to(torch.bfloat16)

    t["embed"] = torch.randn(cfg.vocab_size, H, generator=g, device=device).to(torch.bfloat16)
    for i, l in enumerate(cfg.layers):
        p, c = f"l{i}.", l.mixer
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if l.ff else ()):
            vec(p + n, H, 0.1)
        if l.ff:
            mat(p + "mlp.gate", l.ff, H), mat(p + "mlp.up", l.ff, H), mat(p + "mlp.down", H, l.ff)
        p, h = p + "mix.", c["heads"]
        mat(p + "o", H, h * c["vdim"])
        if l.type == "latent_attention":
            mat(p + "q", h * (c["dim"] + c["rot_dim"]), H), mat(p + "dkv", c["kv_rank"] + c["rot_dim"], H)
            vec(p + "dkv.norm", c["kv_rank"], 0.1, 1.0)
            mat(p + "uk", h * c["dim"], c["kv_rank"]), mat(p + "uv", h * c["vdim"], c["kv_rank"])
            vec(p + "sink", h, 1.0)
            continue
        for n, d in (("q", c["dim"]), ("k", c["dim"]), ("v", c["vdim"]), ("g", c["vdim"])):
            mat(p + n, h * d, H)
        if l.type == "gla":
            vec(p + "norm", c["vdim"], 0.1, 1.0)
            mat(p + "a1", low_rank, H), mat(p + "a2", h * c["dim"], low_rank), vec(p + "a2.b", h * c["dim"], 0.5, 2.0)
        else:
            vec(p + "norm", h * c["vdim"], 0.1, 1.0)
            mat(p + "i", h, H), vec(p + "i.b", h, 0.5, -2.0), mat(p + "f", h, H), vec(p + "f.b", h, 0.5, 4.0)
    vec("final.norm", H, 0.1)
    mat("head", cfg.vocab_size, H)
    return t


def assemble_gidisun_weights(cfg: GidisunConfig, tensors: Dict[str, torch.Tensor], device, dtype, rank: int = 0,
                             world: int = 1) -> GidisunWeights:
    """Checkpoint tensors -> fused, tensor-parallel runtime weights: a layer's input projections are stacked into one matrix,
    heads and feed-forward rows are sharded, norm weights, biases and sinks are kept in fp32."""
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
    lin = lambda *parts: LinearWeight(dev(torch.cat(parts, 0) if len(parts) > 1 else parts[0]))
    by_cols = lambda t: LinearWeight(dev(share(t.t()).t()))
    unit = lambda name: f32(get(name, H).to(torch.float32) + 1.0)          # stored around zero

    subs: List[Sublayer] = []
    mixers = []
    for i, l in enumerate(cfg.layers):
        p, c = f"l{i}.", l.mixer
        m, h = p + "mix.", c["heads"]
        if h % world:
            raise ValueError(f"layer {i}: {h} heads cannot be shared by {world} ranks")
        hl, dk, dv = h // world, c["dim"], c["vdim"]
        o = by_cols(get(m + "o", H, h * dv))
        if l.type == "latent_attention":
            R, dr = c["kv_rank"], c["rot_dim"]
            mask, scaling = c.get("mask") or {}, c["rot"].get("scaling")
            shape = LatentShape(hl, dk, dr, dv, R, float(c["scale"]), int(mask.get("size") or 0), eps)
            rot = rotary_table(c["rot"]["dims"], c["rot"]["base"], YarnScaling(**{k: scaling[k] for k in ("factor", "original", "fast", "slow")})
                               if scaling else None).to(device)
            uv = dev(heads(get(m + "uv", h * dv, R), h)).view(hl, dv, R)
            w = LatentWeights(norm=f32(get(m + "dkv.norm", R)), uk=dev(heads(get(m + "uk", h * dk, R), h)).view(hl, dk, R), uv=uv,
                              uv_t=uv.transpose(1, 2).contiguous(), sink=f32(share(get(m + "sink", h))) if m + "sink" in tensors else None)
            mixer = LatentAttention(i, shape, rot, lin(heads(get(m + "q", h * (dk + dr), H), h), get(m + "dkv", R + dr, H)), w, o)
        else:
            main = [heads(get(m + n, h * d, H), h) for n, d in (("q", dk), ("k", dk), ("v", dv), ("g", dv))]
            if l.type == "gla":
                a1 = get(m + "a1", None, H)
                mixer = GatedLinearAttention(i, hl, dk, dv, float(c["tau"]), eps, lin(*main, a1),
                                             dev(heads(get(m + "a2", h * dk, a1.shape[0]), h)), f32(heads(get(m + "a2.b", h * dk), h)),
                                             f32(get(m + "norm", dv)), o)
            else:
                mixer = MLstm(i, hl, dk, dv, float(c["gate_cap"]), eps, lin(*main, share(get(m + "i", h, H)), share(get(m + "f", h, H))),
                              f32(share(get(m + "i.b", h))), f32(share(get(m + "f.b", h))), f32(heads(get(m + "norm", h * dv), h)), o)
        mixers.append(mixer)
        subs.append(Sublayer(mixer, unit(p + "norm1"), unit(p + "norm1b")))
        if l.ff:
            ff = DenseFeedForward(i, lin(share(get(p + "mlp.gate", l.ff, H)), share(get(p + "mlp.up", l.ff, H))),
                                  by_cols(get(p + "mlp.down", H, l.ff)))
            subs.append(Sublayer(ff, unit(p + "norm2"), unit(p + "norm2b")))
    head = get("head", cfg.vocab_size, H)
    return GidisunWeights(embed=dev(get("embed", cfg.vocab_size, H)), sublayers=subs, mixers=mixers, final_norm=unit("final.norm"),
                          lm_head=LinearWeight(dev(share(head))), vocab_offset=rank * (cfg.vocab_size // world))


class GidisunModel(DecoderStack):
    def __init__(self, cfg: GidisunConfig, weights: GidisunWeights, ctx: Optional[ParallelContext] = None, ops=None,
                 comm: Optional[Comm] = None):
        self.cfg, self.w = cfg, weights
        ctx = ctx or ParallelContext(device=weights.embed.device)
        dtype = weights.embed.dtype
        self.specs = [m.spec for m in weights.mixers]
        self.sublayers = [Sublayer(functools.partial(s.run, self), s.norm, s.post_norm) for s in weights.sublayers]
        self._init_stack(ctx, ops or get_ops(cfg, ctx.device, ctx, dtype), comm, dtype)

    @classmethod
    def from_tensors(cls, cfg: GidisunConfig, tensors: Dict[str, torch.Tensor], ctx: Optional[ParallelContext] = None,
                     dtype=torch.bfloat16) -> "GidisunModel":
        ctx = ctx or ParallelContext()
        w = assemble_gidisun_weights(cfg, tensors, ctx.device, dtype, ctx.rank if ctx.world > 1 else 0, ctx.world)
        return cls(cfg, w, ctx)


def load_gidisun_model(model_dir: str, ctx: Optional[ParallelContext] = None, dtype=torch.bfloat16):
    """(cfg, model) from a directory of config.json and safetensors shards."""
    from ..checkpoint.safetensors_io import load_dir
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = GidisunConfig.from_dict(json.load(f))
    return cfg, GidisunModel.from_tensors(cfg, load_dir(model_dir), ctx, dtype)
