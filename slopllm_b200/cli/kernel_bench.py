"""Kernel micro-benchmarks at the production shapes of one rank of a TP-8 GLM-5-class model.

    python -m slopllm_b200.cli.kernel_bench [--cases linear,mlp,moe,gemm,fp8,mixers] [--tokens 1,8,32,4096] [--iters 20]

For every (kernel, token count) it prints one JSON line with the device time (CUDA events, median of `--iters`
runs, three warm-up runs, a 256 MB write between runs so that no operand is served from L2), the algorithmic
bytes and FLOPs, and both as fractions of the measured roofline (`MEASURED_PEAKS.json` in the working
directory, or `--peaks <file>`; otherwise 6650 GB/s and 1590 TFLOP/s and the line says "fallback").

The reference's counterparts are `tests/python/bench_gemv.py`, `tests/python/bench_nvfp4_mul_mat_id.py`,
`tests/python/bench_indexer_decode.py` and `tests/python/bench_indexer_prefill.py` (the attention / indexer
kernels are covered by `slopllm_b200.cli.profile_step --op-times`, which times them inside a real step).
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
from typing import Callable, Dict, List, Tuple

import torch

FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


def load_peaks(path: str | None = None) -> Dict[str, float]:
    """Roofline denominators: measured copy bandwidth (GB/s) and bf16 GEMM throughput (TFLOP/s)."""
    for p in ([path] if path else []) + ["MEASURED_PEAKS.json"]:
        if p and os.path.exists(p):
            with open(p) as f:
                d = json.load(f)
            return {"hbm_gbs": float(d["hbm_gbs"]), "bf16_tflops": float(d["bf16_tflops"]), "source": "measured"}
    return dict(FALLBACK_PEAKS)


def roofline_row(name: str, tokens: int, us: float, nbytes: float, flops: float, peaks: Dict[str, float]) -> Dict:
    """One result line: achieved bandwidth / throughput and the fraction of the slower-bound roofline."""
    t_mem = nbytes / (peaks["hbm_gbs"] * 1e9)
    t_mma = flops / (peaks["bf16_tflops"] * 1e12)
    bound = "memory" if t_mem >= t_mma else "tensor"
    floor_us = 1e6 * max(t_mem, t_mma)
    return {"kernel": name, "tokens": tokens, "us": round(us, 2), "gbytes_s": round(nbytes / us / 1e3, 1),
            "tflops": round(flops / us / 1e6, 2), "bound": bound, "roofline_us": round(floor_us, 2),
            "fraction_of_roofline": round(floor_us / us, 3), "peaks": peaks["source"]}


def linear_shapes(cfg, tp: int) -> List[Tuple[str, int, int, bool]]:
    """(name, out features, in features, nvfp4) of one rank's linears."""
    hl = cfg.num_attention_heads // tp
    qkv_rows = cfg.q_lora_rank + cfg.kv_lora_rank + cfg.qk_rope_head_dim + cfg.index_head_dim + cfg.index_n_heads
    qb_rows = hl * (cfg.qk_nope_head_dim + cfg.qk_rope_head_dim) + cfg.index_n_heads * cfg.index_head_dim
    return [
        ("qkv_a_bf16", qkv_rows, cfg.hidden_size, False),
        ("q_b_bf16", qb_rows, cfg.q_lora_rank, False),
        ("o_proj", cfg.hidden_size, hl * cfg.v_head_dim, bool(cfg.quant_o_proj)),
        ("dense_gate_up", 2 * cfg.intermediate_size // tp, cfg.hidden_size, bool(cfg.quant_dense_mlp)),
        ("dense_down", cfg.hidden_size, cfg.intermediate_size // tp, bool(cfg.quant_dense_mlp)),
        ("lm_head_bf16", cfg.vocab_size // tp, cfg.hidden_size, False),
    ]


def weight_bytes(n: int, k: int, nvfp4: bool) -> int:
    return n * k // 2 + n * k // 16 if nvfp4 else 2 * n * k


def time_op(fn: Callable[[], object], iters: int, flush: torch.Tensor) -> float:
    """Median device time in microseconds; `flush` (larger than L2) is rewritten before every timed run."""
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
        times.append(1e3 * a.elapsed_time(b))
    return statistics.median(times)


def mixer_rows(emit, tokens, iters: int, flush, peaks, dev, h: int = 16, dk: int = 128, dv: int = 128, rank: int = 512, rot: int = 64,
               window: int = 1024, context: int = 2048, n_kv: int = 4) -> None:
    """Token mixers of the hybrid families at 16 heads of 128: talking-heads attention, token shift, retention, minGRU, attention with turned values, channel-wise delta rule,
    windowed grouped-query attention, GLA, mLSTM and latent attention beside Gated DeltaNet and paged grouped-query attention.  More than 64 tokens: one prompt; fewer: that many sequences of `context` tokens decode one each."""
    import types
    from ..models.glm_moe_dsa import StepState
    from ..ops import delta as DL, delta_chunk as DC, dense as D, get_ops, grouped as G, latent as L, recurrent as RC, shift as SH, talking as TK
    from ..ops.rotary import AngleTable, rotary_table
    ops = get_ops(types.SimpleNamespace(rms_norm_eps=1e-6), dev)
    g = torch.Generator(device=dev).manual_seed(3)
    rnd = lambda *s, k=1.0: torch.randn(*s, device=dev, generator=g) * k
    bf = lambda *s, k=1.0: rnd(*s, k=k).to(torch.bfloat16)
    for T in tokens:
        prompt = T > 64
        B = 1 if prompt else T
        start = 0 if prompt else context - 1
        kv = T if prompt else context
        width = -(-kv // 64)
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
        pt = torch.arange(B * width, dtype=torch.int32, device=dev).view(B, width)
        st = StepState(input_ids=torch.zeros(T, dtype=torch.int64, device=dev), positions=i32([start + i if prompt else start for i in range(T)]),
                       batch_idx=i32([0 if prompt else i for i in range(T)]), page_table=pt, max_kv_len=kv)
        qo = i32([0, T] if prompt else list(range(T + 1)))
        if prompt:
            st.extra.update(spans=[[0, T]], qo_indptr=qo, max_q=T)
        sidx, plan = i32(list(range(B))), RC.ChunkPlan.of(st)
        low16, S = rnd(T, 16), rnd(B, h, dk, dv)
        io = T * h * (2 * dk + 3 * dv) * 2 + 2 * B * h * dk * dv * 4
        flops = 4.0 * T * h * dk * dv
        a2, a2b, nw, nwh = bf(h * dk, 16), rnd(h * dk), rnd(dv), rnd(h * dv)
        proj, projf = bf(T, h * 2 * (dk + dv)), rnd(T, h * 2 * (dk + dv))
        pr = proj if prompt else projf                        # decoding rows arrive in fp32
        io += 0 if prompt else T * h * (2 * dk + 2 * dv) * 2
        us = time_op(lambda: RC.gla_mix(pr, low16, a2, a2b, 16.0, nw, 1e-6, S, qo, sidx, h, dk, dv, torch.bfloat16, plan), iters, flush)
        emit(roofline_row("gla", T, us, io, flops, peaks))
        gates, ib, fb = rnd(T, 2 * h), rnd(h), rnd(h) + 4
        state = (S, rnd(B, h, dk), torch.zeros(B, h, device=dev))
        us = time_op(lambda: RC.mlstm_mix(pr, gates, ib, fb, 15.0, nwh, 1e-6, state, qo, sidx, h, dk, dv, torch.bfloat16, plan), iters, flush)
        emit(roofline_row("mlstm", T, us, io, flops, peaks))
        # retention, minGRU, attention with whole-row norms and turned values, norm of the sum, biased activation
        angle = AngleTable()
        turn, v_turn = angle.turn(dk, 1e4), angle.turn(dv, 1e4)
        angles, rout = angle.of(st), bf(T, h * dv)
        us = time_op(lambda: angle.at(st.positions), iters, flush)
        emit(roofline_row("angle_table", T, us, T * (angles.shape[1] * 8 + 4), 0.0, peaks))
        decay = RC.retention_decays([1 - 2.0 ** (-5 - i % 6) for i in range(h)]).to(dev)
        us = time_op(lambda: RC.retention_mix(pr, decay, turn, angles, 1e-6, S, qo, sidx, h, dk, dv, rout, 1.0, plan), iters, flush)
        emit(roofline_row("retention", T, us, io, flops, peaks))
        W = h * dv
        gru, gb, gS = (bf if prompt else rnd)(T, 3 * W), rnd(2 * W), rnd(B, W)
        us = time_op(lambda: RC.min_gru_mix(gru, gb, gS, qo, sidx, W, torch.bfloat16, plan), iters, flush)
        emit(roofline_row("min_gru", T, us, T * W * (3 * (2 if prompt else 4) + 2) + 8 * B * W, 0.0, peaks))
        rs = G.GroupedShape(h, n_kv, 128, 128, 128 ** -0.5, eps=1e-6)
        rw = G.RowNormWeights(rnd(h * 128), rnd(n_kv * 128), rnd((h + 2 * n_kv) * 128), rnd(h))
        rproj, rk, rv = (bf if prompt else rnd)(T, (h + 2 * n_kv) * 128), bf(B * width * 64, n_kv, 128), bf(B * width * 64, n_kv, 128)
        us = time_op(lambda: G.grouped_row_pre(rproj, rs, rw, turn, v_turn, angles, st, rk, rv, torch.bfloat16), iters, flush)
        emit(roofline_row("grouped_row_pre", T, us, T * 128 * (h + 2 * n_kv) * (2 + (2 if prompt else 4)), 0.0, peaks))
        rq = G.grouped_row_pre(rproj, rs, rw, turn, v_turn, angles, st, rk, rv, torch.bfloat16)
        us = time_op(lambda: G.grouped_attention(rq, rs, rw, st, rk, rv, rout, G.Finish(v_turn, angles, 1.0)), iters, flush)
        every = T * (T + 1) / 2 if prompt else T * kv
        emit(roofline_row("grouped_attention (full context, turned values)", T, us, 2.0 * (T if prompt else T * kv) * n_kv * 256 + 4.0 * T * h * 128,
                          4.0 * every * h * 128, peaks))
        H, sy = h * 128, rnd(T, h * 128)
        sb, sres = rnd(H), rnd(T, H)
        us = time_op(lambda: ops.sum_norm(sy, sres, 2.0, sb, sb, None, 1e-6), iters, flush)
        emit(roofline_row("sum_norm", T, us, T * H * 14.0, 0.0, peaks))
        gu, act, ab2 = bf(T, 8 * H), bf(T, 4 * H), rnd(8 * H)
        us = time_op(lambda: ops.gated_act(gu, act, "gelu_tanh", ab2), iters, flush)
        emit(roofline_row("gated_act (gelu, biases)", T, us, T * H * 24.0, 0.0, peaks))
        us = time_op(lambda: ops.silu_mul(gu, act), iters, flush)
        emit(roofline_row("gated_act (silu)", T, us, T * H * 24.0, 0.0, peaks))
        qkv, ab = bf(T, h * (2 * dk + dv)), bf(T, h)
        us = time_op(lambda: RC.gdn_scan(qkv, ab, ab, ib, fb, S, qo, sidx, h, dk, dv), iters, flush)
        emit(roofline_row("gdn (scan alone)", T, us, T * h * (2 * dk + 2 * dv) * 2 + 2 * B * h * dk * dv * 4, flops, peaks))
        # gated delta rule with a decay per key channel (low ranks of 128, four taps)
        ds = DL.DeltaShape(h, h, dk, dv, 4, 1e-6)
        dw = DL.DeltaWeights(rnd(4, ds.channels), bf(h * dk, 128, k=0.09), bf(h * dv, 128, k=0.09), rnd(h * dk) - 3, rnd(h) * 0.5, nw)
        dmain, fine, ring = (bf if prompt else rnd)(T, ds.channels), rnd(T, 256 + h), torch.zeros(B, 4, ds.channels, device=dev)
        dout = bf(T, h * dv)
        us = time_op(lambda: DL.channel_delta_mix(dmain, fine, ds, dw, S, ring, st, qo, sidx, dout, ops, plan), iters, flush)
        low = 2.0 * T * 128 * h * (dk + dv)
        emit(roofline_row("channel_delta (convolutions, low-rank gates, recurrence)", T, us,
                          T * ds.channels * (2 if prompt else 4) + T * (256 + h) * 4 + T * h * dv * 2 + 2 * B * h * dk * dv * 4 + h * (dk + dv) * 256
                          + (0 if prompt else 2 * B * ds.channels * 16), 3 * flops / 2 + low, peaks))
        if prompt:
            zf, gt = rnd(T, h * dk), bf(T, h * dv)
            us = time_op(lambda: DC.run_chunks(dmain, zf, gt, fine[:, 256:], ds, dw, S, qo, sidx, dout, plan), iters, flush)
            emit(roofline_row("channel_delta recurrence (3 launches)", T, us, T * (ds.channels * 2 + h * (dk * 4 + dv * 4)) + 2 * h * dk * dv * 4,
                              3 * flops / 2, peaks))
            us = time_op(lambda: DL.short_conv(dmain, dw.conv, ring, st.positions, qo, sidx, T, torch.bfloat16), iters, flush)
            emit(roofline_row("short_conv", T, us, 4.0 * T * ds.channels, 0.0, peaks))
            cw, cs = bf(ds.channels, 4), torch.zeros(B, ds.channels, 3, device=dev)
            us = time_op(lambda: RC.causal_conv1d(dmain, cw, None, cs, qo, sidx), iters, flush)
            emit(roofline_row("causal_conv1d (sequential)", T, us, 4.0 * T * ds.channels, 0.0, peaks))
        # windowed grouped-query attention whose values are its keys
        gs = G.GroupedShape(h, n_kv, 128, 128, 128 ** -0.5, window, 4, 1e-6, own_values=False)
        gw = G.GroupedWeights(rnd(128), rnd(128), rnd(h))
        gproj, gk, gv, gout = (bf if prompt else rnd)(T, (h + n_kv) * 128), bf(B * width * 64, n_kv, 128), bf(B * width * 64, n_kv, 128), bf(T, h * 128)
        table = rotary_table(128, 1e6).to(dev)
        us = time_op(lambda: G.grouped_pre(gproj, gs, gw, table, st, gk, gv, torch.bfloat16), iters, flush)
        emit(roofline_row("grouped_pre", T, us, T * 128 * ((h + n_kv) * (2 if prompt else 4) + 2 * (h + 2 * n_kv)), 0.0, peaks))
        gq = G.grouped_pre(gproj, gs, gw, table, st, gk, gv, torch.bfloat16)
        us = time_op(lambda: G.grouped_attention(gq, gs, gw, st, gk, gv, gout), iters, flush)
        seen = sum(min(start + i + 1, window + 4) for i in range(T)) if prompt else T * min(kv, window + 4)
        emit(roofline_row("grouped_attention (window)", T, us, 2.0 * (T if prompt else seen) * n_kv * 256 + 4.0 * T * h * 128, 4.0 * seen * h * 128, peaks))
        # attention
        sh = L.LatentShape(h, dk, rot, dv, rank, (dk + rot) ** -0.5, window)
        uv = bf(h, dv, rank, k=rank ** -0.5)
        w = L.LatentWeights(rnd(rank), bf(h, dk, rank, k=rank ** -0.5), uv, uv.transpose(1, 2).contiguous(), rnd(h))
        rt = rotary_table(rot, 1e6).to(dev)
        cache, qd = bf(B * width * 64, sh.row), bf(T, h * (dk + rot) + sh.row)
        us = time_op(lambda: L.latent_pre(qd, sh, w, rt, st, cache), iters, flush)
        emit(roofline_row("latent_pre", T, us, 2 * T * (2 * h * rot + 2 * sh.row), 0.0, peaks))
        q_rot = L.latent_pre(qd, sh, w, rt, st, cache)
        pairs = sum(min(start + i + 1, window) for i in range(T)) if prompt else T * min(kv, window)
        if prompt:
            out = bf(T, h * dv)
            us = time_op(lambda: L.latent_prefill(qd, q_rot, sh, w, st, cache, ops, out), iters, flush)
            fl = 2.0 * pairs * h * (dk + rot + dv) + 2.0 * T * rank * h * (dk + dv)
            emit(roofline_row("latent_prefill (gather, expand, attend)", T, us, 2.0 * T * (sh.row + h * (dk + rot + dv)), fl, peaks))
            rows, k, v = bf(T, sh.row), bf(T, h * dk), bf(T, h * dv)
            pp = L.PortionPlan.of(st, window)
            us = time_op(lambda: L.portion_attention(qd, dk + rot, q_rot, k, v, pp, out, heads=h, h0=0, group=h, dim=dk, vdim=dv, window=window,
                                                     scale=sh.scale, sink=w.sink, rot_dim=rot, rows=rows, rank=rank), iters, flush)
            emit(roofline_row("latent_prefill kernel", T, us, 2.0 * T * h * (2 * (dk + dv) + rot), 2.0 * pairs * h * (dk + rot + dv), peaks))
        else:
            us = time_op(lambda: L.latent_attention(qd, q_rot, sh, w, st, cache, ops), iters, flush)
            nb = 2.0 * T * min(kv, window) * sh.row + 2.0 * h * rank * (dk + dv)
            emit(roofline_row("latent_decode (absorb, attend, expand)", T, us, nb, 2.0 * pairs * h * (2 * rank + rot), peaks))
        kc, vc = bf(B * width * 64, n_kv, 128), bf(B * width * 64, n_kv, 128)
        q = bf(T, h, 128)
        us = time_op(lambda: D.paged_attention(q, kc, vc, st.positions, st.batch_idx, pt, 64, 128 ** -0.5, qo_indptr=qo if prompt else None,
                                               max_q=T, max_kv_len=kv), iters, flush)
        full = T * (T + 1) / 2 if prompt else T * kv
        emit(roofline_row("paged_attention (full context)", T, us, 2.0 * (T if prompt else T * kv) * n_kv * 256 + 4.0 * T * h * 128,
                          4.0 * full * h * 128, peaks))
        qk = bf(T, (h + 2 * n_kv) * 128)
        us = time_op(lambda: D.qk_norm_rope_cache(qk[:, :h * 128], qk[:, h * 128:(h + n_kv) * 128], qk[:, (h + n_kv) * 128:], None, None, st.positions,
                                                  st.batch_idx, pt, 64, kc, vc, h, n_kv, 128, 64, 1e6, 1e-6), iters, flush)
        emit(roofline_row("qk_norm_rope_cache", T, us, 4 * T * (h + 2 * n_kv) * 128, 0.0, peaks))
        # talking heads in chunks and over the whole context, the join with the token shift, the activation of an ungated feed-forward
        for what, chunk in (("chunk", window), ("full context", 0)):
            ts = TK.TalkingShape(h, n_kv, h, n_kv, 128, 128, 128 ** -0.5, chunk, 1e-6)
            tw = TK.TalkingWeights(rnd((h + 2 * n_kv) * 128), torch.eye(h, device=dev) + rnd(h, h, k=0.1).to(torch.bfloat16).float(), torch.ones(128, device=dev))
            if chunk:
                tq = TK.talking_pre(rproj, ts, tw, st, rk, rv, torch.bfloat16)
                us = time_op(lambda: TK.talking_pre(rproj, ts, tw, st, rk, rv, torch.bfloat16), iters, flush)
                emit(roofline_row("talking_pre", T, us, T * 128 * (h + 2 * n_kv) * (2 + (2 if prompt else 4)), 0.0, peaks))
            us = time_op(lambda: TK.talking_attention(tq, ts, tw, st, rk, rv, rout), iters, flush)
            seen = sum(int(x) - TK.first_visible(int(x), chunk) + 1 for x in st.positions.tolist())
            emit(roofline_row(f"talking_attention ({what})", T, us, 2.0 * (T if prompt else seen) * n_kv * 256 + 4.0 * T * h * 128,
                              2.0 * seen * h * (256 + h), peaks))
        H = h * 128
        y, res, wf, mix = rnd(T, H), rnd(T, H), rnd(H), rnd(H)
        shift = SH.Shift(mix, rnd(B, H), qo, sidx, st.batch_idx)
        us = time_op(lambda: SH.add_shift_norm(st, y, res, wf, 1e-6, shift, torch.bfloat16), iters, flush)
        emit(roofline_row("shift_norm", T, us, T * H * 14.0 + 8 * B * H, 0.0, peaks))
        up = bf(T, 4 * H)
        us = time_op(lambda: ops.plain_act(up, act, "gelu_tanh"), iters, flush)
        emit(roofline_row("plain_act (gelu)", T, us, T * H * 16.0, 0.0, peaks))
        # norms
        H = h * 128
        y, res, wf, wb = rnd(T, H), rnd(T, H), rnd(H), bf(H)
        us = time_op(lambda: ops.post_norm(y, res, wf, wf, 1e-6), iters, flush)
        emit(roofline_row("post_norm", T, us, T * H * 14.0, 0.0, peaks))
        us = time_op(lambda: ops.add_rmsnorm(y, res, wb, 1e-6), iters, flush)
        emit(roofline_row("add_rmsnorm", T, us, T * H * 14.0, 0.0, peaks))


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="slopllm_b200.cli.kernel_bench")
    ap.add_argument("--cases", default="linear,mlp,moe")
    ap.add_argument("--tokens", default="1,8,32,4096")
    ap.add_argument("--tp-shape", type=int, default=8)
    ap.add_argument("--iters", type=int, default=20)
    ap.add_argument("--peaks", default=None)
    args = ap.parse_args(argv)
    from ..config import GlmMoeDsaConfig
    from ..models.weights import _gen, _rand_linear, random_layer
    from ..ops.cuda_ops import CudaOps
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    peaks = load_peaks(args.peaks)
    cfg = GlmMoeDsaConfig.glm5(num_layers=4)
    ops = CudaOps(cfg)
    tokens = [int(t) for t in args.tokens.split(",")]
    cases = set(args.cases.split(","))
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    g = _gen(1, dev)
    rows = []

    def emit(r):
        rows.append(r)
        print(json.dumps(r), flush=True)

    if "linear" in cases:
        for name, n, k, fp4 in linear_shapes(cfg, args.tp_shape):
            w = _rand_linear(n, k, g, dev, torch.bfloat16, fp4)
            for T in tokens:
                x = torch.randn(T, k, device=dev, generator=g).to(torch.bfloat16)
                us = time_op(lambda: ops.linear(x, w), args.iters, flush)
                emit(roofline_row(name + ("_nvfp4" if fp4 else ""), T, us, weight_bytes(n, k, fp4) + 2 * T * (n + k), 2.0 * T * n * k, peaks))
            del w
    if "gemm" in cases:
        # the tcgen05 GEMM itself (bf16 weights of every linear's shape) at both tile widths, and the two grouped expert
        # GEMMs of a prefill chunk (rows sorted by expert, 8 routes per token)
        from ..ops import tcgen05
        from ..ops.gemm import grouped_gemm
        for T in [t for t in tokens if t > 32]:
            for name, n, k, _ in linear_shapes(cfg, args.tp_shape):
                w = (torch.randn(n, k, device=dev, generator=g) * 0.02).to(torch.bfloat16)
                x = torch.randn(T, k, device=dev, generator=g).to(torch.bfloat16)
                for bn in (128, 256):
                    us = time_op(lambda: tcgen05.gemm_bf16(x, w, False, bn), args.iters, flush)
                    emit(roofline_row(f"gemm_bn{bn}_{name}", T, us, 2.0 * (n * k + T * (n + k)), 2.0 * T * n * k, peaks))
                del w, x
            E, I, Hh = cfg.n_routed_experts, cfg.moe_intermediate_size // args.tp_shape, cfg.hidden_size
            nrows = T * cfg.num_experts_per_tok
            cnt = torch.bincount(torch.randint(0, E, (nrows,), device=dev, generator=g), minlength=E)
            off = torch.zeros(E + 1, dtype=torch.int32, device=dev)
            off[1:] = torch.cumsum(cnt, 0).to(torch.int32)
            for name, n, k in (("grouped_gate_up", 2 * I, Hh), ("grouped_down", Hh, I)):
                w = (torch.randn(E, n, k, device=dev, generator=g) * 0.02).to(torch.bfloat16)
                a = torch.randn(nrows, k, device=dev, generator=g).to(torch.bfloat16)
                for bn in (128, 256):
                    us = time_op(lambda: grouped_gemm(a, w, off, False, bn), args.iters, flush)
                    emit(roofline_row(f"{name}_bn{bn}", T, us, 2.0 * (E * n * k + nrows * (n + k)), 2.0 * nrows * n * k, peaks))
                del w, a
    if "fp8" in cases:
        # FP8 block-scaled projections of a Qwen3-8B-class dense model kept in FP8 (one byte per weight streamed)
        from ..models.weights import LinearWeight
        from ..ops import dense as D
        for name, n, k in (("fp8_qkv", 6144, 4096), ("fp8_o_proj", 4096, 4096), ("fp8_gate_up", 24576, 4096), ("fp8_down", 4096, 12288)):
            q, sc = D.fp8_block_quantize(torch.randn(n, k, device=dev, generator=g) * 0.05)
            w = LinearWeight(q, fp8_scale=sc)
            for T in tokens:
                x = torch.randn(T, k, device=dev, generator=g).to(torch.bfloat16)
                us = time_op(lambda: ops.linear(x, w), args.iters, flush)
                emit(roofline_row(name, T, us, n * k + 4 * sc.numel() + 2 * T * (n + k), 2.0 * T * n * k, peaks))
            del w, q
    if "mixers" in cases:
        mixer_rows(emit, tokens, args.iters, flush, peaks, dev)
    if "experts" in cases:
        # small bf16 experts (softmax routing) of a 2048-wide model, 32 of 2048 and 128 of 768 with 4 and 8 a token
        from ..models.weights import ExpertWeights
        from ..ops import experts as EX
        for E, top, I, Hh in ((32, 4, 2048, 2048), (128, 8, 768, 2048)):
            r = lambda *s: (torch.randn(*s, device=dev, generator=g) * s[-1] ** -0.5).to(torch.bfloat16)
            ex = ExpertWeights(r(E, 2 * I, Hh), r(E, Hh, I))
            for T in tokens:
                x, z, out = r(T, Hh) * Hh ** 0.5, torch.randn(T, E, device=dev, generator=g), torch.zeros(T, Hh, device=dev)
                ids, wts = EX.route_softmax(z, top, 4, 2)
                us = time_op(lambda: EX.route_softmax(z, top, 4, 2), args.iters, flush)
                emit(roofline_row(f"route_softmax_{E}", T, us, 4.0 * T * E, 0.0, peaks))
                us = time_op(lambda: EX.add_experts(x, ex, ids, wts, out, ops), args.iters, flush)
                uniq = int(torch.unique(ids).numel())
                row = roofline_row(f"experts_{E}x{I}", T, us, uniq * 3 * I * Hh * 2 + T * Hh * 10, 6.0 * T * top * I * Hh, peaks)
                row["experts_touched"] = uniq
                emit(row)
                z2, c2 = torch.randn(T, E + 8, device=dev, generator=g), torch.randn(E + 8, device=dev, generator=g) * 0.02
                us = time_op(lambda: EX.route_softmax(z2, top, correction=c2), args.iters, flush)
                emit(roofline_row(f"route_softmax_{E}+8 (corrected)", T, us, 4.0 * T * (E + 8), 0.0, peaks))
                ids, wts = EX.route_softmax(z2, top, correction=c2)
                us = time_op(lambda: EX.add_experts(x, ex, ids, wts, out, ops, True), args.iters, flush)
                real = int((ids < E).sum())
                row = roofline_row(f"experts_{E}x{I} beside 8 identity experts", T, us,
                                   int(torch.unique(ids[ids < E]).numel()) * 3 * I * Hh * 2 + T * Hh * 10, 6.0 * real * I * Hh, peaks)
                emit(row)
            del ex
    H = cfg.hidden_size
    if "mlp" in cases:
        lw = random_layer(cfg, 0, 0, dev, torch.bfloat16, 0, args.tp_shape, exact=False)
        nb = lw.mlp_w13.nbytes() + lw.mlp_w2.nbytes()
        nk = lw.mlp_w13.out_features * lw.mlp_w13.in_features + lw.mlp_w2.out_features * lw.mlp_w2.in_features
        for T in tokens:
            x = torch.randn(T, H, device=dev, generator=g).to(torch.bfloat16)
            us = time_op(lambda: ops.dense_mlp(x, lw), args.iters, flush)
            emit(roofline_row("dense_mlp_layer", T, us, nb + 4 * T * H, 2.0 * T * nk, peaks))
        del lw
    if "moe" in cases:
        lw = random_layer(cfg, 3, 0, dev, torch.bfloat16, 0, args.tp_shape, exact=False)
        ex = lw.experts
        E = ex.w13.shape[0]
        per_expert = (ex.w13.numel() + ex.w2.numel() + ex.s13.numel() + ex.s2.numel()) // E if ex.is_nvfp4 else 2 * (ex.w13.numel() + ex.w2.numel()) // E
        per_expert_mac = (ex.w13.shape[1] * H + H * ex.inter)
        shared = 0 if lw.shared is None else per_expert * lw.shared.inter // ex.inter
        for T in tokens:
            x = torch.randn(T, H, device=dev, generator=g).to(torch.bfloat16)
            ids, _ = ops.route(x, lw)
            uniq = int(torch.unique(ids).numel())
            us = time_op(lambda: ops.moe_tp(x, lw), args.iters, flush)
            nbytes = uniq * per_expert + shared + lw.router_w.numel() * 2 + 4 * T * H
            flops = 2.0 * T * (cfg.num_experts_per_tok + (1 if lw.shared is not None else 0)) * per_expert_mac + 2.0 * T * E * H
            r = roofline_row("moe_layer", T, us, nbytes, flops, peaks)
            r["experts_touched"] = uniq
            emit(r)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
