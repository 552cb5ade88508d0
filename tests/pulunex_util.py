"""Shared pieces of the Pulunex tests: configurations, engines."""
import torch

import pulunex_oracle as O
from gidisun_util import feed, portions, random_ids, row_error      # noqa: F401  (schedules are the same for every family)
from slopllm_b200.models.pulunex import PulunexConfig, PulunexModel
from slopllm_b200.parallel.dist import ParallelContext
from slopllm_b200.runtime.engine import Engine


def configs():
    """name -> raw configuration."""
    return {
        # sizes that no vector load or tensor-core tile divides; a layer without a feed-forward, one over another's keys with its own chunk
        "odd": O.config([O.layer(6, 3, 9, 14, size=37, scale=0.41, mlp=O.dense(35)), O.layer(6, 2, 11, 7, mlp=O.moe(5, 2, 13, identity=3, shared=9)),
                         O.layer(4, 2, 11, 7, size=50, kv_from=1), O.layer(3, 3, 6, 10, size=19, mlp=O.moe(3, 3, 7))],
                        width=45, vocab=101, eps=1e-4, embed_scale=0.6, logit_scale=1.7, positions=300),
        # whole 16-byte rows: tensor-core kernels, ragged tiles, chunks that are no multiple of a page or tile
        "tiled": O.config([O.layer(6, 2, 40, 24, size=72, mlp=O.moe(7, 3, 24, identity=2, shared=40)), O.layer(12, 4, 32, 64, size=100, mlp=O.dense(88)),
                           O.layer(8, 4, 32, 64, size=33, scale=0.3, kv_from=1, mlp=O.moe(6, 2, 16, shared=24)),
                           O.layer(12, 4, 32, 64, kv_from=1, mlp=O.moe(9, 2, 32, identity=4)), O.layer(5, 5, 24, 16, size=64)],
                          width=80, vocab=163, embed_scale=1.4, logit_scale=0.35, positions=512),
        # every count that can be one, every factor 1; a chunk of a single position
        "ones": O.config([O.layer(1, 1, 8, 2, size=1, scale=1.0, mlp=O.dense(1)), O.layer(1, 1, 2, 1, scale=1.0, mlp=O.moe(1, 1, 1)),
                          O.layer(1, 1, 2, 1, kv_from=1, mlp=O.moe(1, 1, 8, identity=1, shared=1))], width=16, vocab=19, positions=256),
        # many heads: three and four blocks of 16, one key head, values wider than keys and than 128
        "wide": O.config([O.layer(40, 4, 16, 136, size=90, scale=0.2, mlp=O.dense(64)), O.layer(20, 1, 64, 200, mlp=O.moe(20, 6, 16, identity=12, shared=8)),
                          O.layer(64, 8, 24, 16, size=130, scale=0.1), O.layer(32, 32, 16, 16, size=48)], width=128, vocab=257, positions=512),
    }


def make_engine(raw, tensors, device="cpu", dtype=torch.float32, num_pages=24, max_batch=4, max_states=4, cuda_graph=True, ctx=None):
    ctx = ctx or ParallelContext(device=torch.device(device, 0) if device == "cuda" else torch.device(device))
    cfg = PulunexConfig.from_dict(raw)
    model = PulunexModel.from_tensors(cfg, tensors, ctx, dtype)
    return Engine(cfg, model, num_pages=num_pages, max_batch=max_batch, max_seq_len=num_pages * 64, cuda_graph=cuda_graph,
                  max_states=max_states)


def sharp_model():
    """Few, long chunks and sharp scores, so that tokens hundreds of positions back decide."""
    raw = O.config([O.layer(4, 2, 24, 32, size=200, scale=0.9, mlp=O.dense(48)), O.layer(4, 2, 24, 32, scale=0.8, mlp=O.moe(4, 2, 24, identity=1, shared=16)),
                    O.layer(4, 2, 24, 32, size=256, scale=0.9, kv_from=1)], width=64, vocab=131, positions=512)
    return raw, O.random_tensors(raw, 4)


def same(got, want):
    """fp32 rounding only."""
    return bool(row_error(got, want).max() < 2e-5)
