"""Shared pieces of the Vononex tests: configurations, engines."""
import torch

import vononex_oracle as O
from gidisun_util import feed, portions, random_ids, row_error      # noqa: F401  (schedules are the same for every family)
from slopllm_b200.models.vononex import VononexConfig, VononexModel
from slopllm_b200.parallel.dist import ParallelContext
from slopllm_b200.runtime.engine import Engine


def configs():
    """name -> raw configuration."""
    return {
        # sizes no vector load or tensor-core tile divides; partial rotations; values wider than keys; layers without a feed-forward
        "odd": O.config([O.parallel_layer(heads=6, kv_heads=3, dim=9, vdim=14, dims=6, base=500.0, scale=0.41, left_scale=0.6, right_scale=1.7,
                                          r_heads=5, r_dim=10, r_vdim=7, r_dims=4, r_base=900.0, ff=35),
                         O.mingru_layer(width=37), O.mingru_layer(width=30, ff=18), O.parallel_layer(heads=2, kv_heads=1, dim=12, vdim=6, r_heads=1, r_dim=13,
                                                                                                  r_vdim=22, r_dims=12)], width=44, vocab=101, eps=1e-4, alpha=1.6),
        # whole 16-byte rows: tensor-core and chunked kernels, ragged last tiles, layers that differ in everything
        "tiled": O.config([O.mingru_layer(width=104, ff=88),
                           O.parallel_layer(heads=6, kv_heads=2, dim=40, vdim=24, dims=24, base=5e5, left_scale=1.3, right_scale=0.8, r_heads=3, r_dim=48, r_vdim=72,
                                            r_dims=32, r_base=300.0, decay=[0.9, 0.99, 0.998], ff=64),
                           O.parallel_layer(heads=5, kv_heads=5, dim=24, vdim=40, scale=0.3, left_scale=-0.7, right_scale=1.1, r_heads=4, r_dim=24, r_vdim=16,
                                            decay=[1.0, 0.5, 0.75, 0.999]),
                           O.mingru_layer(width=56)], width=80, vocab=163, alpha=2.5),
        # every count that can be one, every factor 1
        "ones": O.config([O.parallel_layer(heads=1, kv_heads=1, dim=8, vdim=2, dims=2, scale=1.0, r_heads=1, r_dim=8, r_vdim=8, r_dims=2, decay=[0.0], ff=8),
                          O.mingru_layer(width=1, ff=1), O.parallel_layer(heads=1, kv_heads=1, dim=2, vdim=2, r_heads=1, r_dim=2, r_vdim=1)],
                         width=16, vocab=19, alpha=1.0),
        # heads wider than 128, many heads on one key head, recurrences wider than the model
        "wide": O.config([O.parallel_layer(heads=20, kv_heads=1, dim=64, vdim=136, base=1e6, r_heads=2, r_dim=136, r_vdim=160, r_dims=128, ff=96),
                          O.parallel_layer(heads=3, kv_heads=3, dim=160, vdim=200, dims=64, r_heads=6, r_dim=64, r_vdim=96),
                          O.mingru_layer(width=264, ff=64)], width=128, vocab=257),
        # no attention, so no paged rows at all
        "recurrent": O.config([O.mingru_layer(width=24, ff=40), O.mingru_layer(width=72)], width=48, vocab=61, alpha=0.5),
    }


def make_engine(raw, tensors, device="cpu", dtype=torch.float32, num_pages=24, max_batch=4, max_states=4, cuda_graph=True, ctx=None):
    ctx = ctx or ParallelContext(device=torch.device(device, 0) if device == "cuda" else torch.device(device))
    cfg = VononexConfig.from_dict(raw)
    model = VononexModel.from_tensors(cfg, tensors, ctx, dtype)
    return Engine(cfg, model, num_pages=num_pages, max_batch=max_batch, max_seq_len=num_pages * 64, cuda_graph=cuda_graph,
                  max_states=max_states)


def far_key_model():
    """Sharp attention and nearly undamped recurrences, so that tokens hundreds of positions back stay in the logits."""
    raw = configs()["tiled"]
    raw["layers"][1]["mixer"]["right"]["decay"] = [0.999, 0.9995, 0.998]
    t = O.random_tensors(raw, 4)
    for i in (0, 3):
        t[f"l{i}.mix.z.b"] = t[f"l{i}.mix.z.b"] - 4
    for i in (1, 2):
        t[f"l{i}.mix.left.temp"] = t[f"l{i}.mix.left.temp"] * 2
    return raw, t


def same(got, want):
    """fp32 rounding only.  A retention head's output is divided by its own size, so a token whose query and key almost cancel (the first
    ones of a sequence have little else to sum) shows rounding enlarged: single rows get more room than the mean."""
    err = row_error(got, want)
    return bool(err.mean() < 5e-6 and err.max() < 3e-4)
