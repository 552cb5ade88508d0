"""`model_type` -> loader and capabilities.  Reference: `src/model_registry.ts:1-56`."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Dict, Optional, Tuple

import torch

from ..parallel.dist import ParallelContext


@dataclass
class ModelRegistration:
    phased_prefill: bool
    context_parallel: bool
    mtp: bool
    persistent_loader: bool
    load: Callable            # (model_dir, ctx, mtp[, dtype]) -> (cfg, model)
    float32: bool = False     # also runs entirely in fp32 on a GPU (`load` then takes `dtype`)
    kernel_sources: Optional[Tuple[str, ...]] = None     # csrc/*.cu that serve the family (None: the complete library)


def _load_glm_moe_dsa(model_dir: str, ctx: ParallelContext, mtp: int = 0):
    from ..checkpoint.loader import load_model
    from ..parallel.fused import make_comm
    from .glm_moe_dsa import GlmMoeDsaModel
    dtype = torch.bfloat16 if ctx.device.type == "cuda" else torch.float32
    tp_world = ctx.world          # weights stay tensor-parallel under context parallelism too
    cfg, w = load_model(model_dir, ctx.device, dtype, ctx.rank if tp_world > 1 else 0, tp_world, ep=ctx.ep, with_mtp=mtp > 0)
    return cfg, GlmMoeDsaModel(cfg, w, ctx, comm=make_comm(ctx, cfg))


def _load_dense(model_dir: str, ctx: ParallelContext, mtp: int = 0):
    from .dense import load_dense_model
    return load_dense_model(model_dir, ctx)


def _load_glm5_next(model_dir: str, ctx: ParallelContext, mtp: int = 0):
    from .glm5_next import Glm5NextModel
    m = Glm5NextModel.from_pretrained(model_dir, ctx)
    return m.cfg, m


def _load_gidisun(model_dir: str, ctx: ParallelContext, mtp: int = 0, dtype=None):
    from .gidisun import load_gidisun_model
    if dtype is None:
        dtype = torch.bfloat16 if ctx.device.type == "cuda" else torch.float32
    return load_gidisun_model(model_dir, ctx, dtype)


def _load_zemezen(model_dir: str, ctx: ParallelContext, mtp: int = 0, dtype=None):
    from .zemezen import load_zemezen_model
    if dtype is None:
        dtype = torch.bfloat16 if ctx.device.type == "cuda" else torch.float32
    return load_zemezen_model(model_dir, ctx, dtype)


def _load_vononex(model_dir: str, ctx: ParallelContext, mtp: int = 0, dtype=None):
    from .vononex import load_vononex_model
    if dtype is None:
        dtype = torch.bfloat16 if ctx.device.type == "cuda" else torch.float32
    return load_vononex_model(model_dir, ctx, dtype)


def _load_pulunex(model_dir: str, ctx: ParallelContext, mtp: int = 0, dtype=None):
    from .pulunex import load_pulunex_model
    if dtype is None:
        dtype = torch.bfloat16 if ctx.device.type == "cuda" else torch.float32
    return load_pulunex_model(model_dir, ctx, dtype)


MODEL_REGISTRY: Dict[str, ModelRegistration] = {
    "glm_moe_dsa": ModelRegistration(True, True, True, True, _load_glm_moe_dsa),
    "glm5_next": ModelRegistration(False, False, False, True, _load_glm5_next),
    "qwen3": ModelRegistration(False, False, False, True, _load_dense),
    "qwen3_5": ModelRegistration(False, False, False, False, _load_dense),
    "gidisun": ModelRegistration(False, False, False, False, _load_gidisun, float32=True,
                                 kernel_sources=("elementwise", "gated_chunk", "gated_scan", "gemm_tcgen05", "gemv", "latent_attn", "latent_mma", "linear_simt",
                                                 "sampling", "sandwich_norm", "sparse_mla")),
    "zemezen": ModelRegistration(False, False, False, False, _load_zemezen, float32=True,
                                 kernel_sources=("delta_chunk", "delta_step", "elementwise", "gemm_tcgen05", "gemv", "grouped_attn", "latent_attn", "latent_mma",
                                                 "linear_simt", "moe_sort", "moe_stream", "parallel_block", "sampling", "sandwich_norm",
                                                 "short_conv", "sparse_mla")),
    "vononex": ModelRegistration(False, False, False, False, _load_vononex, float32=True,
                                 kernel_sources=("elementwise", "gated_chunk", "gated_scan", "gemm_tcgen05", "gemv", "grouped_attn", "latent_mma", "linear_simt",
                                                 "min_gru", "parallel_block", "rotary", "sampling", "sandwich_norm")),
    "pulunex": ModelRegistration(False, False, False, False, _load_pulunex, float32=True,
                                 kernel_sources=("elementwise", "gemm_tcgen05", "gemv", "grouped_attn", "linear_simt", "moe_sort", "moe_stream", "parallel_block",
                                                 "sampling", "sandwich_norm", "talking_attn", "token_shift")),
}


HYBRID_FAMILIES = ("gidisun", "zemezen", "vononex", "pulunex")      # assembled from the shared mixers


@dataclass
class HybridFamily:
    config: type              # with `from_dict` (config.json) and `tiny`
    model: type               # with `from_tensors`
    random_tensors: Callable  # cfg -> checkpoint tensors
    plan: Callable            # memory plan, `utils/sizing.py`


def hybrid_family(name: str) -> Optional[HybridFamily]:
    """The parts of a hybrid family by model type or a spec that starts with it ("zemezen-tiny"); None for other families."""
    import importlib
    from ..utils import sizing
    for f in HYBRID_FAMILIES:
        if name.startswith(f):
            m = importlib.import_module(f".{f}", __package__)
            return HybridFamily(getattr(m, f.capitalize() + "Config"), getattr(m, f.capitalize() + "Model"), getattr(m, f"random_{f}_tensors"),
                                getattr(sizing, f"plan_{f}"))
    return None


def checkpoint_config_dir(model_dir: str) -> str:
    """A CSF container keeps the model's config under `metadata/`."""
    if not os.path.isfile(os.path.join(model_dir, "config.json")) and os.path.isfile(os.path.join(model_dir, "metadata", "config.json")):
        return os.path.join(model_dir, "metadata")
    return model_dir


def inspect_model(model_dir: str, cp: bool = False, mtp: int = 0):
    """(model_type, registration, raw config) with the option checks of the reference's `inspectModel`."""
    path = os.path.join(checkpoint_config_dir(model_dir), "config.json")
    with open(path) as f:
        config = json.load(f)
    mt = config.get("model_type")
    if mt is None and isinstance(config.get("architecture"), str):
        mt = config["architecture"].lower()
    if not isinstance(mt, str) or mt not in MODEL_REGISTRY:
        raise ValueError(f"unsupported model_type {mt!r} in {path}; supported types: {', '.join(MODEL_REGISTRY)}")
    reg = MODEL_REGISTRY[mt]
    if cp and not reg.context_parallel:
        raise ValueError(f"{mt} does not support --cp")
    if mtp > 0 and not reg.mtp:
        raise ValueError(f"{mt} does not support --mtp")
    return mt, reg, config


def load_registered(reg: ModelRegistration, model_dir: str, ctx: ParallelContext, mtp: int = 0, dtype: Optional[str] = None):
    """`dtype`: "bfloat16" / "float32" (None: bfloat16 on a GPU, float32 on the CPU)."""
    if dtype is None or (dtype == "bfloat16") == (ctx.device.type == "cuda"):
        return reg.load(model_dir, ctx, mtp)
    if not reg.float32:
        raise ValueError(f"{model_dir}: this model family does not run in {dtype} on {ctx.device.type}")
    return reg.load(model_dir, ctx, mtp, dtype=getattr(torch, dtype))


def load_any(model_dir: str, ctx: Optional[ParallelContext] = None, mtp: int = 0, dtype: Optional[str] = None):
    ctx = ctx or ParallelContext()
    _, reg, _ = inspect_model(model_dir, cp=ctx.cp, mtp=mtp)
    return load_registered(reg, model_dir, ctx, mtp, dtype)
