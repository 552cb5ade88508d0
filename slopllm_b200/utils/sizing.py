"""Memory plan of a deployment (glm_moe_dsa, and the dense Qwen3 / Qwen3.5 families), computed from the configuration alone
(no weights, no GPU).

`plan_memory` answers the questions that come before a launch: how many bytes of weights does one rank hold under a given
tensor / expert / context parallelism, what does one KV page cost, how many pages fit next to the weights in the device
memory that `--arena` allows, and how much context that is.  The reference answers them with its shape-only backend
(`src/meta_ops.ts`) and the sizing notes in `GLM51-NVFP4-weights.md`; here the same arithmetic is a function and a command
(`python -m slopllm_b200 plan`).
"""
from __future__ import annotations

from dataclasses import asdict, dataclass
from typing import Dict

from ..config import PAGE_SIZE, GlmMoeDsaConfig

GIB = 1 << 30


def _lin(n: int, k: int, nvfp4: bool, elem: int = 2) -> int:
    """Bytes of an [n, k] linear weight: NVFP4 = half a byte per weight + one e4m3 scale per 16 + one fp32 global."""
    return n * k // 2 + n * k // 16 + 4 if nvfp4 else n * k * elem


def layer_weight_bytes(cfg: GlmMoeDsaConfig, layer: int, tp: int = 1, ep: bool = False, elem: int = 2) -> int:
    """Bytes of one decoder layer on one rank: attention projections head-sharded, o_proj / down row-sharded, gate / up
    column-sharded, the small replicated projections and norms whole; with `ep` the routed experts are split by expert
    instead of by intermediate column (the shared expert stays column-sharded)."""
    H, R, Dr = cfg.hidden_size, cfg.kv_lora_rank, cfg.qk_rope_head_dim
    Dn, Dv, Q = cfg.qk_nope_head_dim, cfg.v_head_dim, cfg.q_lora_rank
    hl = cfg.num_attention_heads // tp
    full = cfg.indexer_is_full(min(layer, len(cfg.indexer_types) - 1)) if cfg.indexer_types else False
    Hi, Di = cfg.index_n_heads, cfg.index_head_dim
    qkv_rows = Q + R + Dr + ((Di + Hi) if full else 0)
    qb_rows = hl * (Dn + Dr) + (Hi * Di if full else 0)
    b = _lin(qkv_rows, H, False, elem) + _lin(qb_rows, Q, False, elem)
    b += hl * (Dn + Dv) * R * elem                                    # absorbed k_nope and v projections
    b += _lin(H, hl * Dv, bool(cfg.quant_o_proj), elem)
    b += (2 * H + Q + R + (2 * Di if full else 0)) * elem             # norms
    if cfg.is_moe_layer(layer):
        E, I = cfg.n_routed_experts, cfg.moe_intermediate_size
        q = bool(cfg.quant_experts)
        b += E * H * elem + E * 4                                     # router weight + bias
        if ep:
            b += (E // tp) * (_lin(2 * I, H, q, elem) + _lin(H, I, q, elem))
        else:
            b += E * (_lin(2 * I // tp, H, q, elem) + _lin(H, I // tp, q, elem))
        if cfg.n_shared_experts:
            Is = I * cfg.n_shared_experts // tp
            b += _lin(2 * Is, H, q, elem) + _lin(H, Is, q, elem)
    else:
        I = cfg.intermediate_size // tp
        q = bool(cfg.quant_dense_mlp)
        b += _lin(2 * I, H, q, elem) + _lin(H, I, q, elem)
    return b


def model_weight_bytes(cfg: GlmMoeDsaConfig, tp: int = 1, ep: bool = False, with_mtp: bool = True, elem: int = 2) -> int:
    H, V = cfg.hidden_size, cfg.vocab_size
    n = cfg.num_hidden_layers + (cfg.num_nextn_predict_layers if with_mtp else 0)
    b = V * H * elem + (V // tp) * H * elem + H * elem                # embedding (whole), lm_head shard, final norm
    for i in range(n):
        b += layer_weight_bytes(cfg, i, tp, ep, elem)
        if i >= cfg.num_hidden_layers:                                # MTP layer extras: two norms, eh_proj, head norm
            b += 3 * H * elem + _lin(H, 2 * H, False, elem)
    return b


def kv_page_bytes(cfg: GlmMoeDsaConfig, with_mtp: bool = True) -> int:
    """Bytes one page id costs on one rank: 64 rows per layer of the packed sparse-MLA cache, plus the indexer key rows
    of the layers that own an indexer.  Under context parallelism a page id covers 64 x W tokens and every rank stores 64
    of them, so this figure does not change with W; the tokens per page do."""
    n = cfg.num_hidden_layers + (cfg.num_nextn_predict_layers if with_mtp else 0)
    per_token = 0
    for i in range(n):
        per_token += cfg.kv_row_bytes
        if cfg.indexer_is_full(min(i, len(cfg.indexer_types) - 1)):
            per_token += cfg.index_row_bytes
    return per_token * PAGE_SIZE


def step_workspace_bytes(cfg: GlmMoeDsaConfig, tp: int, chunk: int, context: int, cp: int = 1) -> int:
    """Upper estimate of the transient buffers of one prefill chunk of `chunk` tokens against `context` cached tokens: the
    residual and activation rows, the expert-sorted MoE rows, the sparse-MLA query / output rows, and the indexer's score
    matrix (bounded by its 2 GiB budget)."""
    H, k = cfg.hidden_size, max(1, cfg.num_experts_per_tok)
    hl = max(1, cfg.num_attention_heads // tp) * (cp if cp > 1 else 1)     # CP gathers all heads
    I = max(cfg.moe_intermediate_size, 1) // tp
    act = chunk * H * (4 + 4 + 2 + 2)                                      # residual in / out (fp32), normed x, attention out
    moe = chunk * k * (H * 2 + 2 * I * 2 + I * 2 + H * 2) + chunk * H * 4  # sorted rows, gate/up, act, down rows, fp32 out
    mla = chunk * hl * (cfg.kv_lora_rank + cfg.qk_rope_head_dim) * 2 + chunk * hl * cfg.kv_lora_rank * 4 * 2
    keys = -(-context // max(1, cp))
    scores = min(chunk * keys * 4, 2 * GIB) + chunk * cfg.index_topk * 12
    dense = chunk * 2 * (cfg.intermediate_size // tp) * 2 * 2
    return act + max(moe, dense) + mla + scores


@dataclass
class MemoryPlan:
    tp: int
    cp: int
    ep: bool
    weights_bytes: int
    page_bytes: int
    tokens_per_page: int
    workspace_bytes: int
    budget_bytes: int
    max_pages: int
    max_tokens: int
    requested_pages: int
    requested_fits: bool

    def to_dict(self) -> Dict[str, object]:
        d = asdict(self)
        d.update(weights_gib=round(self.weights_bytes / GIB, 2), workspace_gib=round(self.workspace_bytes / GIB, 2),
                 kv_gib_at_max=round(self.max_pages * self.page_bytes / GIB, 2), budget_gib=round(self.budget_bytes / GIB, 2))
        return d


def plan_memory(cfg: GlmMoeDsaConfig, world: int = 1, cp: bool = False, ep: bool = False, mtp: int = 0, batch_size: int = 8,
                chunk_size: int = 8192, max_pages: int = 0, arena_gb: float = 0.0, device_gb: float = 180.0,
                context: int = 0, reserve_gb: float = 4.0) -> MemoryPlan:
    """The plan for one rank of a `world`-GPU replica.  `arena_gb` (0: `device_gb`) is what the process may allocate;
    `reserve_gb` stays free for the CUDA context, NCCL and the symmetric region.  `context` is the longest sequence the
    workspace estimate assumes (0: the pages asked for, or 64K tokens)."""
    tp = world
    cpw = world if cp else 1
    weights = model_weight_bytes(cfg, tp, ep, with_mtp=mtp > 0)
    page = kv_page_bytes(cfg, with_mtp=mtp > 0)
    tpp = PAGE_SIZE * cpw
    requested = max_pages if max_pages > 0 else batch_size * -(-chunk_size // PAGE_SIZE)
    ctx = context or (max_pages * tpp if max_pages > 0 else 65536)
    work = step_workspace_bytes(cfg, tp, chunk_size, ctx, cpw)
    budget = int(((arena_gb if arena_gb > 0 else device_gb) - reserve_gb) * GIB)
    left = budget - weights - work
    fit = max(0, left // page)
    return MemoryPlan(tp=tp, cp=cpw, ep=ep, weights_bytes=weights, page_bytes=page, tokens_per_page=tpp, workspace_bytes=work,
                      budget_bytes=budget, max_pages=int(fit), max_tokens=int(fit) * tpp, requested_pages=requested,
                      requested_fits=requested <= fit)


# ---- dense families (Qwen3, Qwen3.5) -----------------------------------------------------------------------------------

def dense_weight_bytes(cfg, tp: int = 1, elem: int = 2, fp8: bool = False) -> int:
    """Per-rank weight bytes of a Qwen3 / Qwen3.5 decoder: attention and Gated-DeltaNet projections head-sharded, MLP
    column / row sharded, embedding whole, lm_head vocabulary-sharded.  `fp8`: the attention and MLP projections stay FP8
    (one byte per weight + one fp32 scale per 128 x 128 block)."""
    H, I, hd = cfg.hidden_size, cfg.intermediate_size, cfg.head_dim

    def lin(n, k, quant=False):
        return n * k + (-(-n // 128)) * (-(-k // 128)) * 4 if quant else n * k * elem
    b = cfg.vocab_size * H * elem + H * elem
    b += (cfg.vocab_size // tp) * H * elem                         # the head's shard is materialised even when it is tied
    for kind in cfg.layer_types:
        b += 2 * H * elem                                           # the two layer norms
        b += lin(2 * I // tp, H, fp8) + lin(H, I // tp, fp8)
        if kind == "full_attention":
            qs = hd * (2 if cfg.attn_output_gate else 1)
            hq, hk = cfg.num_attention_heads // tp, max(1, cfg.num_key_value_heads // tp)
            b += lin(hq * qs + 2 * hk * hd, H, fp8) + lin(H, hq * hd, fp8) + 2 * hd * elem      # qkv, o_proj, q/k norms
        else:
            lh, dk, dv = cfg.linear_num_key_heads // tp, cfg.linear_key_head_dim, cfg.linear_value_head_dim
            conv_dim = lh * (2 * dk + dv)
            b += lin(conv_dim + lh * dv + 2 * lh, H) + lin(H, lh * dv)                          # in-projection, out-projection
            b += conv_dim * cfg.linear_conv_kernel_dim * elem + 2 * lh * 4 + dv * elem          # conv, A_log, dt_bias, norm
    return b


def dense_kv_page_bytes(cfg, tp: int = 1, elem: int = 2) -> int:
    """Bytes of one 64-token page on one rank: K and V rows of every full-attention layer (recurrent layers keep their
    state per sequence, not per page)."""
    n_kv = max(1, cfg.num_key_value_heads // tp)
    full = sum(1 for k in cfg.layer_types if k == "full_attention")
    return full * 2 * n_kv * cfg.head_dim * elem * PAGE_SIZE


def plan_dense(cfg, world: int = 1, batch_size: int = 8, chunk_size: int = 8192, max_pages: int = 0, arena_gb: float = 0.0,
               device_gb: float = 180.0, fp8: bool = False, reserve_gb: float = 4.0) -> MemoryPlan:
    """`plan_memory` for the dense families (tensor parallel only; the workspace estimate is the residual / activation rows
    plus the MLP's gate-up rows of one chunk)."""
    weights = dense_weight_bytes(cfg, world, fp8=fp8)
    page = max(1, dense_kv_page_bytes(cfg, world))
    requested = max_pages if max_pages > 0 else batch_size * -(-chunk_size // PAGE_SIZE)
    work = chunk_size * (cfg.hidden_size * 12 + 2 * (cfg.intermediate_size // world) * 4
                         + (cfg.num_attention_heads // world) * cfg.head_dim * 8)
    budget = int(((arena_gb if arena_gb > 0 else device_gb) - reserve_gb) * GIB)
    fit = max(0, (budget - weights - work) // page)
    return MemoryPlan(tp=world, cp=1, ep=False, weights_bytes=weights, page_bytes=page, tokens_per_page=PAGE_SIZE,
                      workspace_bytes=work, budget_bytes=budget, max_pages=int(fit), max_tokens=int(fit) * PAGE_SIZE,
                      requested_pages=requested, requested_fits=requested <= fit)


# ---- Gidisun --------------------------------------------------------------------------------------------------------------

def gidisun_weight_bytes(cfg, tp: int = 1, elem: int = 2, low_rank: int = 16) -> int:
    """Per-rank weight bytes: projections head-sharded, feed-forward sharded, embedding whole, head vocabulary-sharded; norm
    weights, biases and sinks are fp32.  `low_rank`: width of the GLA decay projection (a tensor shape, not in the
    configuration)."""
    H = cfg.hidden_size
    b = cfg.vocab_size * H * elem + (cfg.vocab_size // tp) * H * elem + 4 * H
    for l in cfg.layers:
        c, h = l.mixer, l.mixer["heads"] // tp
        dk, dv = c["dim"], c["vdim"]
        b += h * dv * H * elem + 4 * 2 * H * (2 if l.ff else 1) + 3 * (l.ff // tp) * H * elem
        if l.type == "latent_attention":
            R, dr = c["kv_rank"], c["rot_dim"]
            b += (h * (dk + dr) + R + dr) * H * elem + h * (dk + 2 * dv) * R * elem + 4 * (R + h)     # (values in two layouts)
        elif l.type == "gla":
            b += (h * 2 * (dk + dv) + low_rank) * H * elem + h * dk * (low_rank * elem + 4) + 4 * dv
        else:
            b += (h * 2 * (dk + dv) + 2 * h) * H * elem + 4 * (2 * h + h * dv)
    return b


def gidisun_cache_bytes(cfg, tp: int = 1, elem: int = 2):
    """(bytes of one 64-token page, bytes of one sequence's recurrent state) on one rank."""
    page = state = 0
    for l in cfg.layers:
        c = l.mixer
        if l.type == "latent_attention":
            page += (c["kv_rank"] + c["rot_dim"]) * elem * PAGE_SIZE
        else:
            h = c["heads"] // tp
            state += 4 * h * (c["dim"] * c["vdim"] + (c["dim"] + 1 if l.type == "mlstm" else 0))
    return page, state


def plan_gidisun(cfg, world: int = 1, batch_size: int = 8, chunk_size: int = 8192, max_pages: int = 0, arena_gb: float = 0.0,
                 device_gb: float = 180.0, elem: int = 2, reserve_gb: float = 4.0) -> MemoryPlan:
    """`plan_memory` for Gidisun (tensor parallel only)."""
    row = max(max(3 * l.ff, 6 * l.mixer["heads"] * (l.mixer["dim"] + l.mixer["vdim"])) for l in cfg.layers) // world
    return _plan_hybrid(cfg, gidisun_weight_bytes(cfg, world, elem), *gidisun_cache_bytes(cfg, world, elem), row, world, batch_size, chunk_size,
                        max_pages, arena_gb, device_gb, elem, reserve_gb)


def _plan_hybrid(cfg, weights: int, page: int, state: int, row: int, world: int, batch_size: int, chunk_size: int, max_pages: int, arena_gb: float,
                 device_gb: float, elem: int, reserve_gb: float) -> MemoryPlan:
    """Plan of a model with paged rows and per-sequence states.  The workspace estimate is the widest layer's rows of one chunk
    (`row` values a token), the recurrent state of every slot, and the transient keys, values and chunk states of a prefill."""
    requested = max_pages if max_pages > 0 else batch_size * -(-chunk_size // PAGE_SIZE)
    work = chunk_size * (cfg.hidden_size * 12 + row * elem) + state * max(64, batch_size) + (1 << 30)
    budget = int(((arena_gb if arena_gb > 0 else device_gb) - reserve_gb) * GIB)
    fit = max(0, (budget - weights - work) // max(1, page))
    return MemoryPlan(tp=world, cp=1, ep=False, weights_bytes=weights, page_bytes=page, tokens_per_page=PAGE_SIZE,
                      workspace_bytes=work, budget_bytes=budget, max_pages=int(fit), max_tokens=int(fit) * PAGE_SIZE,
                      requested_pages=requested, requested_fits=requested <= fit)


# ---- Zemezen --------------------------------------------------------------------------------------------------------------

def zemezen_weight_bytes(cfg, tp: int = 1, elem: int = 2, low_rank: int = 16) -> int:
    """Per-rank weight bytes, as :func:`gidisun_weight_bytes`; experts are sharded like a feed-forward, a layer that uses another's
    weights has none.  `low_rank`: width of the decay and gate projections (tensor shapes, not in the configuration)."""
    H = cfg.hidden_size
    b = cfg.vocab_size * H * elem + (cfg.vocab_size // tp) * H * elem + 4 * H
    for l in cfg.layers:
        if l.weights_of is not None:
            continue
        c, h, dk = l.mixer, l.mixer["heads"] // tp, l.mixer["dim"]
        kv, dv = c.get("kv_heads", c["heads"]) // tp, c.get("vdim", dk)
        b += 4 * H + h * dv * H * elem + 3 * (l.ff // tp) * H * elem
        if l.experts is not None:
            b += l.experts.count * (3 * (l.experts.ff // tp) + 1) * H * elem
        if l.type == "attention":
            b += (h + kv) * dk * H * elem + 4 * (2 * dk + h)
        elif l.type == "latent_attention":
            R = c["kv_rank"]
            b += (h * dk + R) * H * elem + h * (dk + 2 * dv) * R * elem + 4 * R                       # (values in two layouts)
        else:
            rows = 2 * kv * dk + h * dv
            b += (rows + 2 * low_rank + h) * H * elem + h * (dk + dv) * low_rank * elem + 4 * (rows * c["conv"] + h * dk + h + dv)
    return b


def zemezen_cache_bytes(cfg, tp: int = 1, elem: int = 2):
    """(bytes of one 64-token page, bytes of one sequence's recurrent state) on one rank."""
    page = state = 0
    for l in cfg.layers:
        c = l.mixer
        if l.type == "attention":
            page += 2 * (c["kv_heads"] // tp) * c["dim"] * elem * PAGE_SIZE
        elif l.type == "latent_attention":
            page += c["kv_rank"] * elem * PAGE_SIZE
        else:
            h, kv = c["heads"] // tp, c["kv_heads"] // tp
            state += 4 * (h * c["dim"] * c["vdim"] + c["conv"] * (2 * kv * c["dim"] + h * c["vdim"]))
    return page, state


def plan_zemezen(cfg, world: int = 1, batch_size: int = 8, chunk_size: int = 8192, max_pages: int = 0, arena_gb: float = 0.0,
                 device_gb: float = 180.0, elem: int = 2, reserve_gb: float = 4.0) -> MemoryPlan:
    """`plan_memory` for Zemezen (tensor parallel only)."""
    def width(l):
        experts = 0 if l.experts is None else l.experts.top * (3 * l.experts.ff + 2 * cfg.hidden_size * world)
        return max(3 * l.ff, experts) + 8 * l.mixer["heads"] * (l.mixer["dim"] + l.mixer.get("vdim", l.mixer["dim"]))
    return _plan_hybrid(cfg, zemezen_weight_bytes(cfg, world, elem), *zemezen_cache_bytes(cfg, world, elem), max(width(l) for l in cfg.layers) // world,
                        world, batch_size, chunk_size, max_pages, arena_gb, device_gb, elem, reserve_gb)


# ---- Vononex --------------------------------------------------------------------------------------------------------------

def vononex_weight_bytes(cfg, tp: int = 1, elem: int = 2) -> int:
    """Per-rank weight bytes, as :func:`gidisun_weight_bytes`; heads, channels and feed-forward rows are sharded with their fp32 biases,
    norms and decays."""
    H = cfg.hidden_size
    b = cfg.vocab_size * H * elem + (cfg.vocab_size // tp) * H * elem + 4 * H
    for l in cfg.layers:
        c, ff = l.mixer, l.ff // tp
        b += 4 * H + 3 * ff * H * elem + (4 * (2 * H + 2 * ff) if ff else 0)
        if l.type == "mingru":
            W = c["width"] // tp
            b += 4 * W * H * elem + 4 * 2 * W
            continue
        a, r = c["left"], c["right"]
        h, kv, hr = a["heads"] // tp, a["kv_heads"] // tp, r["heads"] // tp
        qk = (h + kv) * a["dim"]
        b += (qk + (h + kv) * a["vdim"]) * H * elem + 4 * (2 * qk + kv * a["vdim"] + h + H)
        b += hr * (2 * r["dim"] + 3 * r["vdim"]) * H * elem + 4 * 2 * hr
    return b


def vononex_cache_bytes(cfg, tp: int = 1, elem: int = 2):
    """(bytes of one 64-token page, bytes of one sequence's recurrent state) on one rank."""
    page = state = 0
    for l in cfg.layers:
        c = l.mixer
        if l.type == "mingru":
            state += 4 * (c["width"] // tp)
        else:
            a, r = c["left"], c["right"]
            page += (a["kv_heads"] // tp) * (a["dim"] + a["vdim"]) * elem * PAGE_SIZE
            state += 4 * (r["heads"] // tp) * r["dim"] * r["vdim"]
    return page, state


def plan_vononex(cfg, world: int = 1, batch_size: int = 8, chunk_size: int = 8192, max_pages: int = 0, arena_gb: float = 0.0,
                 device_gb: float = 180.0, elem: int = 2, reserve_gb: float = 4.0) -> MemoryPlan:
    """`plan_memory` for Vononex (tensor parallel only)."""
    def width(l):
        if l.type == "mingru":
            return max(3 * l.ff, 4 * l.mixer["width"])
        a, r = l.mixer["left"], l.mixer["right"]
        return max(3 * l.ff, 3 * a["heads"] * (a["dim"] + a["vdim"]) + r["heads"] * (2 * r["dim"] + 3 * r["vdim"]))
    return _plan_hybrid(cfg, vononex_weight_bytes(cfg, world, elem), *vononex_cache_bytes(cfg, world, elem), max(width(l) for l in cfg.layers) // world,
                        world, batch_size, chunk_size, max_pages, arena_gb, device_gb, elem, reserve_gb)


# ---- Pulunex --------------------------------------------------------------------------------------------------------------

def pulunex_weight_bytes(cfg, tp: int = 1, elem: int = 2) -> int:
    """Per-rank weight bytes, as :func:`gidisun_weight_bytes`; queries and keys are whole on every rank (their scores are mixed), value and
    output heads and feed-forward rows sharded; norms spread over the row, biases, mixtures and corrections are fp32."""
    H = cfg.hidden_size
    b = (cfg.vocab_size + cfg.max_positions) * H * elem + (cfg.vocab_size // tp) * H * elem + 4 * H
    for l in cfg.layers:
        c = l.mixer
        h, kv, d, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
        rows = h * d + (0 if l.kv_from is not None else kv * d + kv // tp * dv)
        b += rows * (H * elem + 4) + 4 * (h // tp * h + d) + h // tp * dv * H * elem + 4 * 2 * H
        if l.ff or l.experts is not None:
            b += 4 * H + 2 * (l.ff // tp) * H * elem
        if l.experts is not None:
            e = l.experts
            n = e.count + e.identity
            b += (3 * e.count * (e.ff // tp) + 3 * (e.shared_ff // tp) + n + (1 if e.shared_ff else 0)) * H * elem + 4 * n
    return b


def pulunex_cache_bytes(cfg, tp: int = 1, elem: int = 2):
    """(bytes of one 64-token page, bytes of one sequence's state) on one rank."""
    page = sum((l.mixer["kv_heads"] * l.mixer["dim"] + l.mixer["kv_heads"] // tp * l.mixer["vdim"]) * elem * PAGE_SIZE
               for l in cfg.layers if l.kv_from is None)
    return page, 4 * cfg.hidden_size * len(cfg.layers)


def plan_pulunex(cfg, world: int = 1, batch_size: int = 8, chunk_size: int = 8192, max_pages: int = 0, arena_gb: float = 0.0,
                 device_gb: float = 180.0, elem: int = 2, reserve_gb: float = 4.0) -> MemoryPlan:
    """`plan_memory` for Pulunex (tensor parallel only)."""
    def width(l):
        e = l.experts
        ff = 2 * l.ff if e is None else 3 * e.shared_ff + e.top * (3 * e.ff + 2 * cfg.hidden_size * world)
        return max(ff, 3 * l.mixer["heads"] * (l.mixer["dim"] * world + l.mixer["vdim"]))
    return _plan_hybrid(cfg, pulunex_weight_bytes(cfg, world, elem), *pulunex_cache_bytes(cfg, world, elem), max(width(l) for l in cfg.layers) // world,
                        world, batch_size, chunk_size, max_pages, arena_gb, device_gb, elem, reserve_gb)
