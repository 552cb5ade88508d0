"""Shared pieces of the Gidisun tests: configurations, engines, schedules."""
import torch

import gidisun_oracle as O
from slopllm_b200.models.gidisun import GidisunConfig, GidisunModel
from slopllm_b200.parallel.dist import ParallelContext
from slopllm_b200.runtime.engine import Engine

YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}


def configs():
    """name -> (raw configuration, low rank of the GLA decay)."""
    return {
        # sizes no vector load or tensor-core tile divides; partial rotation
        "odd": (O.config([O.gla_layer(heads=3, dim=10, vdim=14, tau=5.0, ff=36),
                          O.attention_layer(heads=3, dim=12, rot_dim=10, dims=6, vdim=20, kv_rank=36, window=11, scaling=YARN, scale=0.31),
                          O.mlstm_layer(heads=5, dim=9, vdim=7, cap=6.0, ff=20)], width=44, vocab=101, eps=1e-4), 5),
        # whole 16-byte rows: tensor-core and chunked kernels, ragged last tiles, window above a key tile
        "tiled": (O.config([O.attention_layer(heads=5, dim=24, rot_dim=16, vdim=40, kv_rank=72, window=70, base=5e5, scaling=YARN, ff=88),
                            O.mlstm_layer(heads=3, dim=40, vdim=72, cap=9.0),
                            O.gla_layer(heads=2, dim=48, vdim=24, tau=12.0, ff=64),
                            O.attention_layer(heads=2, dim=16, rot_dim=8, vdim=136, kv_rank=136, window=17)], width=80, vocab=163), 8),
        # every count and constant that can be one
        "ones": (O.config([O.attention_layer(heads=1, dim=8, rot_dim=8, vdim=8, kv_rank=8, window=1, scale=1.0,
                                             scaling={"factor": 1.0, "original": 32, "fast": 4.0, "slow": 1.0}),
                           O.gla_layer(heads=1, dim=8, vdim=8, tau=1.0), O.mlstm_layer(heads=1, dim=8, vdim=8, cap=1.0, ff=8)],
                          width=16, vocab=19), 1),
        # value heads wider than 128, key heads wider than value heads
        "wide": (O.config([O.gla_layer(heads=2, dim=64, vdim=160, tau=16.0), O.mlstm_layer(heads=2, dim=136, vdim=96, ff=96),
                           O.attention_layer(heads=3, dim=64, rot_dim=32, vdim=96, kv_rank=264, window=130, ff=64)], width=128, vocab=257), 16),
    }


def make_engine(raw, tensors, device="cpu", dtype=torch.float32, num_pages=24, max_batch=4, max_states=4, cuda_graph=True, ctx=None):
    ctx = ctx or ParallelContext(device=torch.device(device, 0) if device == "cuda" else torch.device(device))
    cfg = GidisunConfig.from_dict(raw)
    model = GidisunModel.from_tensors(cfg, tensors, ctx, dtype)
    return Engine(cfg, model, num_pages=num_pages, max_batch=max_batch, max_seq_len=num_pages * 64, cuda_graph=cuda_graph,
                  max_states=max_states)


def random_ids(raw, n, seed):
    return torch.randint(0, raw["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def feed(engine, ids, cuts, seq=None):
    """Logits of every position of one sequence fed in the given portions (fp32, CPU)."""
    s = seq or engine.kv.new_sequence()
    out, at = [], 0
    for n in cuts:
        out.append(engine.step([s], [ids[at:at + n]], [range(n)]))
        at += n
    assert at == len(ids)
    if seq is None:
        engine.finish(s)
    return torch.cat(out).cpu()


def portions(total, sizes, tail=0):
    """Cut `total` tokens into the cyclic `sizes`, the last `tail` one by one."""
    out, i, left = [], 0, total - tail
    while left > 0:
        out.append(min(sizes[i % len(sizes)], left))
        left -= out[-1]
        i += 1
    return out + [1] * tail


def row_error(got, want):
    """Root mean square of the difference of each row (mean taken off) over that of the reference."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt())
