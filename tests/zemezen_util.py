"""Shared pieces of the Zemezen tests: configurations, engines."""
import torch

import zemezen_oracle as O
from gidisun_util import feed, portions, random_ids, row_error      # noqa: F401  (schedules are the same for every family)
from slopllm_b200.models.zemezen import ZemezenConfig, ZemezenModel
from slopllm_b200.parallel.dist import ParallelContext
from slopllm_b200.runtime.engine import Engine


def configs():
    """name -> (raw configuration, low ranks of decay and gate)."""
    return {
        # sizes no vector load or tensor-core tile divides; partial rotation; layers without a feed-forward; shared weights
        "odd": (O.config([O.delta_layer(heads=6, kv_heads=2, dim=10, vdim=14, conv=2, mlp=O.moe(9, 4, 12, 3, 2)),
                          O.attention_layer(heads=6, kv_heads=2, dim=12, dims=6, base=500.0, window=11, keep=3, scale=0.31, mlp=O.dense(36)),
                          O.latent_layer(heads=3, dim=12, vdim=20, kv_rank=36), 0,
                          O.attention_layer(heads=2, kv_heads=2, dim=10, window=0, mlp=O.moe(5, 2, 10)), 1], width=44, vocab=101, eps=1e-4), (5, 3)),
        # whole 16-byte rows: tensor-core, chunked and grouped kernels, ragged last tiles, windows above a key tile
        "tiled": (O.config([O.attention_layer(heads=6, kv_heads=2, dim=40, dims=24, window=70, keep=5, base=5e5, mlp=O.moe(10, 3, 32, 5, 3)),
                            O.delta_layer(heads=4, kv_heads=2, dim=24, vdim=40, conv=4, mlp=O.dense(88)),
                            O.latent_layer(heads=5, dim=24, vdim=40, kv_rank=72, mlp=O.moe(6, 2, 48, 2, 1)),
                            O.delta_layer(heads=3, kv_heads=3, dim=48, vdim=16, conv=3), 2, 1], width=80, vocab=163), (8, 16)),
        # every count that can be one
        "ones": (O.config([O.attention_layer(heads=1, kv_heads=1, dim=8, dims=2, window=1, keep=1, scale=1.0, mlp=O.moe(1, 1, 8, 1, 1)),
                           O.delta_layer(heads=1, kv_heads=1, dim=8, vdim=8, conv=1, mlp=O.dense(8)), O.latent_layer(heads=1, dim=8, vdim=8, kv_rank=8)],
                          width=16, vocab=19), (1, 1)),
        # heads wider than 128, many heads on one key head, experts enough for several per lane, a window that keeps more than its size
        "wide": (O.config([O.delta_layer(heads=4, kv_heads=1, dim=136, vdim=160, conv=5, mlp=O.moe(40, 6, 16, 8, 3)),
                           O.attention_layer(heads=20, kv_heads=1, dim=64, window=33, keep=70, base=1e6, mlp=O.dense(96)),
                           O.latent_layer(heads=3, dim=96, vdim=136, kv_rank=264, mlp=O.dense(64)), 1], width=128, vocab=257), (16, 24)),
    }


def make_engine(raw, tensors, device="cpu", dtype=torch.float32, num_pages=24, max_batch=4, max_states=4, cuda_graph=True, ctx=None):
    ctx = ctx or ParallelContext(device=torch.device(device, 0) if device == "cuda" else torch.device(device))
    cfg = ZemezenConfig.from_dict(raw)
    model = ZemezenModel.from_tensors(cfg, tensors, ctx, dtype)
    return Engine(cfg, model, num_pages=num_pages, max_batch=max_batch, max_seq_len=num_pages * 64, cuda_graph=cuda_graph,
                  max_states=max_states)
