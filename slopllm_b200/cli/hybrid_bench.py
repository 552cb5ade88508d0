"""Prefill and decode throughput of the hybrid families side by side: Pulunex, Vononex, Zemezen, Gidisun and Qwen3.5 at equal width, heads,
head sizes and feed-forward, random weights, layers of a real model's size.

    python -m slopllm_b200.cli.hybrid_bench [--sizes small,medium,large] [--batches 1,8,64] [--prompt 4096]

Every stack has four layers with a feed-forward each: three recurrent mixers and one attention layer; Zemezen two of its recurrent
mixers, one windowed and one latent attention layer; Vononex two minGRU layers and two in which attention over the whole context and
retention share the heads (half of them each, so that a layer's projections stay as wide); Pulunex four layers of talking-heads attention in chunks of 1024, one of which uses another's
keys (its dense feed-forward has two matrices, the others' three, so it is half as wide again).  `zemezen_moe` and `pulunex_moe` have 32 experts of a quarter of the feed-forward's width in
every layer, of which a token uses four (Pulunex: of these and four identity experts, beside a shared one of the same width).  Every number is device
time (CUDA events, three warm-up runs, a 256 MB write in front of every timed run so that nothing is served from L2); decode is
a replay of the captured step.  Prints one JSON line; `python bench.py --hybrid [sizes]` prints the same.
"""
from __future__ import annotations

import argparse
import gc
import json
import statistics
import time

import torch

SIZES = {"small": (1024, 4096, 8), "medium": (2048, 8192, 16), "large": (4096, 14336, 32)}      # width, feed-forward, heads of 128
VOCAB, WINDOW = 32768, 1024


def gidisun_config(size: str):
    from ..models.gidisun import GidisunConfig, GidisunLayer
    H, ff, h = SIZES[size]
    attn = {"heads": h, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "scale": 192 ** -0.5, "mask": {"size": WINDOW},
            "rot": {"base": 1e6, "dims": 64, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    gla = {"heads": h, "dim": 128, "vdim": 128, "tau": 16.0}
    mlstm = {"heads": h, "dim": 128, "vdim": 128, "gate_cap": 15.0}
    return GidisunConfig(hidden_size=H, vocab_size=VOCAB, rms_norm_eps=1e-6,
                         layers=[GidisunLayer("gla", gla, ff), GidisunLayer("gla", gla, ff), GidisunLayer("mlstm", mlstm, ff),
                                 GidisunLayer("latent_attention", attn, ff)])


def qwen35_config(size: str):
    from ..models.dense import DenseConfig
    H, ff, h = SIZES[size]
    return DenseConfig(model_type="qwen3_5", hidden_size=H, intermediate_size=ff, num_hidden_layers=4, num_attention_heads=h,
                       num_key_value_heads=max(1, h // 8), head_dim=128, vocab_size=VOCAB, partial_rotary_factor=0.25, attn_output_gate=True,
                       layer_types=["linear_attention"] * 3 + ["full_attention"], linear_num_key_heads=h, linear_key_head_dim=128,
                       linear_num_value_heads=h, linear_value_head_dim=128, gemma_norm=True, weight_prefix="model.language_model.",
                       eos_token_ids=[])


def zemezen_config(size: str, moe: bool = False):
    from ..models.zemezen import ZemezenConfig, ZemezenExperts, ZemezenLayer
    H, ff, h = SIZES[size]
    attn = {"heads": h, "kv_heads": max(1, h // 8), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "rot": {"base": 1e6, "dims": 128},
            "mask": {"size": WINDOW, "keep_first": 4}}
    delta = {"heads": h, "kv_heads": h, "dim": 128, "vdim": 128, "conv": 4}
    latent = {"heads": h, "dim": 128, "vdim": 128, "kv_rank": 512, "scale": 128 ** -0.5}
    mlp = (0, ZemezenExperts(32, 4, ff // 4, 4, 2)) if moe else (ff, None)
    return ZemezenConfig(hidden_size=H, vocab_size=VOCAB, rms_norm_eps=1e-6,
                         layers=[ZemezenLayer("channel_delta", delta, *mlp), ZemezenLayer("channel_delta", delta, *mlp),
                                 ZemezenLayer("attention", attn, *mlp), ZemezenLayer("latent_attention", latent, *mlp)])


def vononex_config(size: str):
    from ..models.vononex import VononexConfig, VononexLayer
    H, ff, h = SIZES[size]
    left = {"heads": h // 2, "kv_heads": max(1, h // 8), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "rot": {"base": 1e6, "dims": 128}}
    right = {"heads": h // 2, "dim": 128, "vdim": 128, "rot": {"base": 1e4, "dims": 128}, "decay": [1 - 2.0 ** (-5 - i % 6) for i in range(h // 2)]}
    pair, gru = {"left": left, "right": right, "left_scale": 1.0, "right_scale": 1.0}, {"width": H}
    return VononexConfig(hidden_size=H, vocab_size=VOCAB, rms_norm_eps=1e-6, alpha=2.0,
                         layers=[VononexLayer("mingru", gru, ff), VononexLayer("parallel", pair, ff), VononexLayer("mingru", gru, ff),
                                 VononexLayer("parallel", pair, ff)])


def pulunex_config(size: str, moe: bool = False):
    from ..models.pulunex import PulunexConfig, PulunexExperts, PulunexLayer
    H, ff, h = SIZES[size]
    c = {"heads": h, "kv_heads": max(1, h // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": WINDOW}}
    mlp = (0, PulunexExperts(32, 4, ff // 4, 4, ff // 4)) if moe else (ff * 3 // 2, None)
    return PulunexConfig(hidden_size=H, vocab_size=VOCAB, rms_norm_eps=1e-6, max_positions=8192,
                         layers=[PulunexLayer("attention", c if i != 3 else {**c, "kv_from": 2}, *mlp) for i in range(4)])


def build(family: str, size: str, ctx):
    if family in ("pulunex", "pulunex_moe"):
        from ..models.pulunex import PulunexModel, random_pulunex_tensors
        cfg = pulunex_config(size, family == "pulunex_moe")
        return cfg, PulunexModel.from_tensors(cfg, random_pulunex_tensors(cfg, 0, device=ctx.device), ctx)
    if family == "vononex":
        from ..models.vononex import VononexModel, random_vononex_tensors
        cfg = vononex_config(size)
        return cfg, VononexModel.from_tensors(cfg, random_vononex_tensors(cfg, 0, device=ctx.device), ctx)
    if family in ("zemezen", "zemezen_moe"):
        from ..models.zemezen import ZemezenModel, random_zemezen_tensors
        cfg = zemezen_config(size, family == "zemezen_moe")
        return cfg, ZemezenModel.from_tensors(cfg, random_zemezen_tensors(cfg, 0, 128, device=ctx.device), ctx)
    if family == "gidisun":
        from ..models.gidisun import GidisunModel, random_gidisun_tensors
        cfg = gidisun_config(size)
        return cfg, GidisunModel.from_tensors(cfg, random_gidisun_tensors(cfg, 0, device=ctx.device), ctx)
    from ..models.dense import DenseModel, random_dense_model
    cfg = qwen35_config(size)
    w, _ = random_dense_model(cfg, 0, ctx.device, torch.bfloat16, draw_device=ctx.device)
    return cfg, DenseModel(cfg, w, ctx)


def median_ms(fn, iters: int, flush: torch.Tensor) -> float:
    for _ in range(3):
        fn()
    times = []
    for _ in range(iters):
        flush.zero_()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        b.synchronize()
        times.append(a.elapsed_time(b))
    return statistics.median(times)


def run_arm(family: str, size: str, batches, prompt: int, iters: int, flush) -> dict:
    from ..ops import tcgen05
    from ..parallel.dist import ParallelContext
    from ..runtime.engine import Engine
    ctx = ParallelContext(device=torch.device("cuda", torch.cuda.current_device()))
    cfg, model = build(family, size, ctx)
    top = max(batches)
    context = min(prompt, 2048)
    pages = -(-(prompt + 64) // 64) + top * (-(-(context + 4 * iters) // 64) + 1)
    eng = Engine(cfg, model, num_pages=pages, max_batch=top, max_seq_len=prompt + 64)
    g = torch.Generator().manual_seed(1)
    out = {"family": family, "size": size, "layers": 4, "params_m": round(_params(model) / 1e6, 1)}
    s = eng.kv.new_sequence()
    ids = torch.randint(0, VOCAB, (prompt,), generator=g).tolist()
    st, _, _ = eng._pack([s], [ids])

    def prefill():
        for name in ("chunk_plan", "portion_plans", "talking_plans", "angles"):
            st.extra.pop(name, None)
        return model.forward_hidden(st, eng.cache)

    ms = median_ms(prefill, iters, flush)
    out["prefill"] = {"tokens": prompt, "ms": round(ms, 3), "tok_s": round(prompt / ms * 1e3)}
    eng.finish(s)
    seqs = [eng.kv.new_sequence() for _ in range(top)]
    for q in seqs:
        eng.prefill([q], [torch.randint(0, VOCAB, (context,), generator=g).tolist()], chunk_size=context)
    out["decode"] = []
    for B in batches:
        last = [1] * B
        for _ in range(3):
            last = eng.decode_step(seqs[:B], last)
        entry = next(e for k, e in eng.graphs.entries.items() if k[0] == "decode" and k[1] == B and e.graph is not None)
        ms = median_ms(entry.graph.replay, iters, flush)
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        for _ in range(iters):
            last = eng.decode_step(seqs[:B], last)
        e2e = (time.perf_counter() - t0) / iters * 1e3
        out["decode"].append({"batch": B, "context": context, "ms": round(ms, 4), "tok_s": round(B / ms * 1e3), "e2e_ms": round(e2e, 4),
                              "kernels": entry.kernels})
    tcgen05.check_errors(ctx.device)
    return out


def _params(model) -> int:
    seen, total, stack = set(), 0, [model.w]
    while stack:
        x = stack.pop()
        if isinstance(x, torch.Tensor):
            if x.data_ptr() not in seen:
                seen.add(x.data_ptr())
                total += x.numel()
        elif isinstance(x, (list, tuple)):
            stack += x
        elif hasattr(x, "func"):                       # functools.partial of a sublayer
            stack += x.args
        elif hasattr(x, "__dataclass_fields__"):
            stack += [getattr(x, f) for f in x.__dataclass_fields__]
    return total


def run(argv=None) -> dict:
    ap = argparse.ArgumentParser(prog="slopllm_b200.cli.hybrid_bench", description=__doc__.split("\n")[0])
    ap.add_argument("--sizes", default="small,medium,large")
    ap.add_argument("--batches", default="1,8,64")
    ap.add_argument("--prompt", type=int, default=4096)
    ap.add_argument("--iters", type=int, default=10)
    ap.add_argument("--families", default="pulunex,pulunex_moe,vononex,zemezen,zemezen_moe,gidisun,qwen3_5")
    args = ap.parse_args(argv)
    torch.cuda.set_device(0)
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    rows = []
    for size in args.sizes.split(","):
        for family in args.families.split(","):
            rows.append(run_arm(family, size, [int(b) for b in args.batches.split(",")], args.prompt, args.iters, flush))
            gc.collect()
            torch.cuda.empty_cache()
    return {"metric": "hybrid_families_prefill_decode", "unit": "tokens/s", "n_gpus": 1, "dtype": "bf16", "data": "synthetic",
            "config": {"vocab": VOCAB, "window": WINDOW, "sizes": {k: dict(zip(("width", "ff", "heads"), v)) for k, v in SIZES.items()},
                       "l2": "256 MB written before every timed run"}, "rows": rows}


def main(argv=None) -> int:
    print(json.dumps(run(argv)), flush=True)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
