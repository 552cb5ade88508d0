"""Vononex: a small decoder whose layers each name a mixer (grouped-query attention beside retention, or a minGRU) and optionally a
feed-forward.  The norm follows the sum, x <- norm(alpha x + sublayer(x)); values turn with their position, queries and keys are
normalised over all heads at once.

This file is the configuration, the checkpoint's tensor names and the assembly of the shared parts: mixers (`models/mixers.py`),
decoder loop and engine hooks (`models/stack.py`), cache (`kv/hybrid.py`).
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
from ..ops.grouped import GroupedShape, RowNormWeights
from ..ops.recurrent import retention_decays
from ..ops.rotary import AngleTable, adjacent_order
from ..parallel.dist import Comm, ParallelContext
from .mixers import GatedFeedForward, MinGru, Retention, RowNormAttention, SideBySide
from .stack import DecoderStack, Sublayer
from .weights import LinearWeight

MIXER_KEYS = {"parallel": ("left", "right", "left_scale", "right_scale"), "mingru": ("width",)}
LEFT_KEYS = ("heads", "kv_heads", "dim", "vdim", "scale", "rot")
RIGHT_KEYS = ("heads", "dim", "vdim", "rot", "decay")


@dataclass
class VononexLayer:
    type: str
    mixer: dict
    ff: int = 0                      # feed-forward width; 0: the layer has none


@dataclass
class VononexConfig:
    hidden_size: int
    vocab_size: int
    rms_norm_eps: float
    alpha: float                     # factor on the residual
    layers: List[VononexLayer]
    eos_token_ids: List[int] = field(default_factory=list)
    model_type: str = "vononex"
    num_nextn_predict_layers: int = 0

    def __post_init__(self):
        if not self.layers:
            raise ValueError("the configuration lists no layers")

        def need(i, what, c, keys):
            missing = [k for k in keys if k not in c]
            if missing:
                raise ValueError(f"layer {i} ({what}): missing {', '.join(missing)}")

        def rotation(i, what, c):
            if c["rot"]["dims"] % 2 or c["rot"]["dims"] > c["dim"]:
                raise ValueError(f"layer {i} ({what}): rot.dims must be even and at most dim")

        for i, l in enumerate(self.layers):
            if l.type not in MIXER_KEYS:
                raise ValueError(f"layer {i}: unknown mixer {l.type!r}")
            need(i, l.type, l.mixer, MIXER_KEYS[l.type])
            if l.type != "parallel":
                continue
            a, r = l.mixer["left"], l.mixer["right"]
            need(i, "left", a, LEFT_KEYS), need(i, "right", r, RIGHT_KEYS)
            rotation(i, "left", a), rotation(i, "right", r)
            if a["heads"] % a["kv_heads"]:
                raise ValueError(f"layer {i}: {a['heads']} heads do not share {a['kv_heads']} key heads evenly")
            if a["vdim"] % 2:
                raise ValueError(f"layer {i}: values turn in pairs, so vdim must be even")
            if len(r["decay"]) != r["heads"]:
                raise ValueError(f"layer {i}: {len(r['decay'])} decays for {r['heads']} heads")

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, raw: dict) -> "VononexConfig":
        layers = []
        for i, l in enumerate(raw["layers"]):
            mlp = l.get("mlp")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            layers.append(VononexLayer(l["type"], dict(l["mixer"]), int(mlp["ff"]) if mlp else 0))
        eos = raw.get("eos_token_id", [])
        return cls(hidden_size=raw["width"], vocab_size=raw["vocab"], rms_norm_eps=raw["norm"]["eps"], alpha=float(raw["postln_alpha"]),
                   layers=layers, eos_token_ids=list(eos) if isinstance(eos, (list, tuple)) else [eos])

    @classmethod
    def tiny(cls) -> "VononexConfig":
        left = {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 32, "scale": 32 ** -0.5, "rot": {"base": 10000.0, "dims": 16}}
        right = {"heads": 4, "dim": 32, "vdim": 48, "rot": {"base": 500000.0, "dims": 32}, "decay": [1 - 2.0 ** -(4 + i) for i in range(4)]}
        pair = {"left": left, "right": right, "left_scale": 0.75, "right_scale": 1.5}
        return cls(hidden_size=128, vocab_size=512, rms_norm_eps=1e-6, alpha=2.0, layers=[
            VononexLayer("parallel", pair, 192), VononexLayer("mingru", {"width": 160}, 192), VononexLayer("parallel", pair)])


@dataclass
class VononexWeights:
    embed: torch.Tensor
    sublayers: List[Sublayer]        # `run` takes the model first
    mixers: list
    angles: AngleTable
    final_norm: torch.Tensor         # fp32
    lm_head: LinearWeight
    vocab_offset: int = 0


def random_vononex_tensors(cfg: VononexConfig, seed: int = 0, device="cpu") -> Dict[str, torch.Tensor]:
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
        vec(p + "norm1", H, 0.1, 1.0)
        if l.ff:
            vec(p + "norm2", H, 0.1, 1.0)
            for n, rows, cols in (("gate", l.ff, H), ("up", l.ff, H), ("down", H, l.ff)):
                mat(f"{p}mlp.{n}", rows, cols), vec(f"{p}mlp.{n}.b", rows, 0.1)
        m = p + "mix."
        if l.type == "mingru":
            W = c["width"]
            mat(m + "z", W, H), vec(m + "z.b", W, 0.5, -1.0), mat(m + "x", W, H), vec(m + "x.b", W, 0.1), mat(m + "g", W, H), mat(m + "o", H, W)
            continue
        a, r = c["left"], c["right"]
        for n, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
            mat(f"{m}left.{n}", rows, H), vec(f"{m}left.{n}.b", rows, 0.1)
            if n != "v":
                vec(f"{m}left.{n}.norm", rows, 0.1, 1.0)
        vec(m + "left.temp", a["heads"], 0.1, 1.0), mat(m + "left.o", H, a["heads"] * a["vdim"]), vec(m + "left.o.b", H, 0.1)
        for n, d in (("q", r["dim"]), ("k", r["dim"]), ("v", r["vdim"]), ("g", r["vdim"])):
            mat(f"{m}right.{n}", r["heads"] * d, H)
        mat(m + "right.o", H, r["heads"] * r["vdim"])
    vec("final.norm", H, 0.1, 1.0)
    mat("head", cfg.vocab_size, H)
    return t


def assemble_vononex_weights(cfg: VononexConfig, tensors: Dict[str, torch.Tensor], device, dtype, rank: int = 0, world: int = 1) -> VononexWeights:
    """Checkpoint tensors -> fused, tensor-parallel runtime weights: a layer's input projections are stacked into one matrix, the
    output projections of mixers that run side by side stand in one; heads, channels and feed-forward rows are sharded; norm weights,
    biases and temperatures are kept in fp32.  Rotated heads are stored with the partners of a rotation side by side
    (`ops/rotary.py: adjacent_order`); the columns of the attention's output projection follow its values."""
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

    def heads(t, h, dims=0):
        """This rank's heads of stacked rows; the first `dims` values of a head in adjacent order."""
        t = share(t.reshape(h, t.shape[0] // h, *t.shape[1:]))
        if dims:
            t = t[:, adjacent_order(t.shape[1], dims).to(t.device)]
        return t.reshape(-1, *t.shape[2:])

    dev = lambda t: t.to(dtype).to(device).contiguous()
    f32 = lambda t: t.to(torch.float32).to(device).contiguous()
    lin = lambda *parts: LinearWeight(dev(torch.cat(parts, 0) if len(parts) > 1 else parts[0]))
    cols = lambda t: share(t.t()).t()

    angles = AngleTable()

    def parallel(i, c):
        """(mixer, bias of its output)"""
        p, a, r = f"l{i}.mix.left.", c["left"], c["right"]
        h, kv, d, dv, rot = a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["rot"]
        if h % world or kv % world or r["heads"] % world:
            raise ValueError(f"layer {i}: {h} heads, {kv} key heads and {r['heads']} retention heads cannot be shared by {world} ranks")
        turn, v_turn = angles.turn(rot["dims"], rot["base"]), angles.turn(dv, rot["base"])
        rows = (("q", h, d, rot["dims"]), ("k", kv, d, rot["dims"]), ("v", kv, dv, dv))
        w = RowNormWeights(f32(heads(get(p + "q.norm", h * d), h, rot["dims"])), f32(heads(get(p + "k.norm", kv * d), kv, rot["dims"])),
                           f32(torch.cat([heads(get(f"{p}{n}.b", u * x), u, k) for n, u, x, k in rows])), f32(share(get(p + "temp", h))))
        left = RowNormAttention(i, GroupedShape(h // world, kv // world, d, dv, float(a["scale"]), eps=eps), turn, v_turn, w, float(c["left_scale"]))
        main = [heads(get(p + n, u * x, H), u, k) for n, u, x, k in rows]
        outs = [heads(get(p + "o", H, h * dv).t(), h, dv).t()]
        bias = f32(get(p + "o.b", H)) * left.scale
        p, h, d, dv, rot = f"l{i}.mix.right.", r["heads"], r["dim"], r["vdim"], r["rot"]
        right = Retention(i, h // world, d, dv, eps, angles.turn(rot["dims"], rot["base"]), retention_decays(share(torch.tensor(r["decay"], dtype=torch.float64)).tolist())
                          .to(device), float(c["right_scale"]))
        gate = [heads(get(p + n, h * x, H), h, k) for n, x, k in (("q", d, rot["dims"]), ("k", d, rot["dims"]), ("v", dv, 0), ("g", dv, 0))]
        outs.append(cols(get(p + "o", H, h * dv)))
        count = lambda parts: sum(t.shape[0] for t in parts)
        return SideBySide(i, "parallel", [left, right], [count(main), count(gate)], [o.shape[1] for o in outs], lin(*main, *gate),
                          LinearWeight(dev(torch.cat(outs, 1)))), bias

    def mingru(i, c):
        p, W = f"l{i}.mix.", c["width"]
        rows = lin(*[share(get(p + n, W, H)) for n in ("z", "x", "g")])
        bias = f32(torch.cat([share(get(p + n + ".b", W)) for n in ("z", "x")]))
        return MinGru(i, W // world, rows, bias, LinearWeight(dev(cols(get(p + "o", H, W))))), None

    subs: List[Sublayer] = []
    mixers = []
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        mixer, bias = {"parallel": parallel, "mingru": mingru}[l.type](i, l.mixer)
        mixers.append(mixer)
        subs.append(Sublayer(mixer, None, f32(get(p + "norm1", H)), cfg.alpha, bias))
        if l.ff:
            m = p + "mlp."
            ff = GatedFeedForward(i, lin(share(get(m + "gate", l.ff, H)), share(get(m + "up", l.ff, H))),
                                  f32(torch.cat([share(get(m + n + ".b", l.ff)) for n in ("gate", "up")])),
                                  LinearWeight(dev(cols(get(m + "down", H, l.ff)))), "gelu_tanh")
            subs.append(Sublayer(ff, None, f32(get(p + "norm2", H)), cfg.alpha, f32(get(m + "down.b", H))))
    head = get("head", cfg.vocab_size, H)
    return VononexWeights(embed=dev(get("embed", cfg.vocab_size, H)), sublayers=subs, mixers=mixers, angles=angles, final_norm=f32(get("final.norm", H)),
                          lm_head=LinearWeight(dev(share(head))), vocab_offset=rank * (cfg.vocab_size // world))


class VononexModel(DecoderStack):
    def __init__(self, cfg: VononexConfig, weights: VononexWeights, ctx: Optional[ParallelContext] = None, ops=None, comm: Optional[Comm] = None):
        self.cfg, self.w = cfg, weights
        ctx = ctx or ParallelContext(device=weights.embed.device)
        dtype = weights.embed.dtype
        self.angles = weights.angles
        self.specs = [m.spec for m in weights.mixers]
        self.sublayers = [dataclasses.replace(s, run=functools.partial(s.run, self)) for s in weights.sublayers]
        self._init_stack(ctx, ops or get_ops(cfg, ctx.device, ctx, dtype), comm, dtype)

    @classmethod
    def from_tensors(cls, cfg: VononexConfig, tensors: Dict[str, torch.Tensor], ctx: Optional[ParallelContext] = None,
                     dtype=torch.bfloat16) -> "VononexModel":
        ctx = ctx or ParallelContext()
        w = assemble_vononex_weights(cfg, tensors, ctx.device, dtype, ctx.rank if ctx.world > 1 else 0, ctx.world)
        return cls(cfg, w, ctx)


def load_vononex_model(model_dir: str, ctx: Optional[ParallelContext] = None, dtype=torch.bfloat16):
    """(cfg, model) from a directory of config.json and safetensors shards."""
    from ..checkpoint.safetensors_io import load_dir
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = VononexConfig.from_dict(json.load(f))
    return cfg, VononexModel.from_tensors(cfg, load_dir(model_dir), ctx, dtype)
