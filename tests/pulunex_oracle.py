"""Plain, slow definition of a Pulunex decoder: whole sequences, fp32 (or fp64) torch, one function per mechanism, no cache and no
kernels.  The tests compare the framework with it; it shares no code with the package.

Also makes small random configurations and checkpoints.
"""
import math

import torch


# ---- mechanisms -----------------------------------------------------------------------------------------------------

def matmul(x, w, b=None):
    y = x @ w.to(x.dtype).t()
    return y if b is None else y + b.to(x.dtype)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def scalar_norm(x, g, eps):
    """RMS norm whose weight is one number."""
    return rms(x, eps) * g.to(x.dtype)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def embed(ids, table, scale, pos):
    """Scaled token vectors plus the learned vectors of positions 0, 1, .."""
    ids = torch.as_tensor(ids)
    return table[ids].to(torch.float32) * scale + pos[:ids.numel()].to(torch.float32)


def token_shift(h, mix, before=None):
    """h_t + (h_{t-1} - h_t) * mix, element by element; `before` stands in front of the first row (None: zeros)."""
    first = torch.zeros_like(h[:1]) if before is None else before[None]
    return h + (torch.cat([first, h[:-1]]) - h) * mix.to(h.dtype)


def chunk_mask(i, j, size):
    """Position i sees j <= i of its own chunk of `size` positions (0: of the whole sequence)."""
    seen = j[None, :] <= i[:, None]
    return seen & (i[:, None] // size == j[None, :] // size) if size else seen


def talking_scores(q, k, scale, talk):
    """Every query head's scores, then a mixture of all heads' for each: q [T, H, D], k [S, H, D] -> [H', T, S] for talk [H', H]."""
    return torch.einsum("gh,hts->gts", talk.to(q.dtype), torch.einsum("thd,shd->hts", q, k) * scale)


def softmax_over(s, mask):
    s = s.masked_fill(~mask, float("-inf"))
    e = torch.exp(s - s.amax(-1, keepdim=True))
    return e / e.sum(-1, keepdim=True)


def keys_values(h, t, p, c, eps):
    T, G = h.shape[0], c["kv_heads"]
    k = rms(matmul(h, t[p + "k"], t[p + "k.b"]).view(T, G, c["dim"]), eps)
    return k, matmul(h, t[p + "v"], t[p + "v.b"]).view(T, G, c["vdim"])


def attention(h, t, p, c, eps, kv):
    """Grouped-query attention with talking heads inside chunks, over the keys and values `kv` (its own or another layer's)."""
    T, H, G = h.shape[0], c["heads"], c["kv_heads"]
    q = rms(matmul(h, t[p + "q"], t[p + "q.b"]).view(T, H, c["dim"]), eps)
    k, v = (x.repeat_interleave(H // G, 1) for x in kv)
    at = torch.arange(T)
    w = softmax_over(talking_scores(q, k, c["scale"], t[p + "talk"]), chunk_mask(at, at, (c.get("mask") or {}).get("size", 0)))
    return matmul(torch.einsum("hts,shv->thv", w, v).reshape(T, -1), t[p + "o"])


def dense_ff(h, t, p):
    return matmul(gelu_tanh(matmul(h, t[p + "up"])), t[p + "down"])


def expert(h, t, p):
    return matmul(silu(matmul(h, t[p + "gate"])) * matmul(h, t[p + "up"]), t[p + "down"])


def choose(z, correction, top):
    """(ids, weights) [T, top]: the largest softmax scores after `correction` was added, weighted by the scores without it."""
    s = torch.softmax(z, -1)
    ids = torch.sort(s + correction.to(s.dtype), dim=-1, descending=True, stable=True).indices[:, :top]
    return ids, s.gather(1, ids)


def mixture(h, t, p, c):
    """Routed experts, of which the last `identity` hand the input through, and a shared expert behind a sigmoid gate."""
    r = c["router"]
    ids, w = choose(matmul(h, t[p + "router"]), t[p + "correction"], r["top"])
    y = torch.zeros_like(h)
    for e in range(r["experts"] + r.get("identity", 0)):
        weight = (w * (ids == e)).sum(-1, keepdim=True)
        y = y + weight * (expert(h, t, f"{p}e{e}.") if e < r["experts"] else h)
    if c.get("shared"):
        y = y + torch.sigmoid(matmul(h, t[p + "shared.sg"])) * expert(h, t, p + "shared.")
    return y


# ---- the model ------------------------------------------------------------------------------------------------------

def residuals(raw, t, ids, dtype=torch.float32):
    """Residual stream after every layer [layers, T, width]."""
    eps = raw["norm"]["eps"]
    x = embed(ids, t["embed"], raw["embedding"]["scale"], t["pos"]).to(dtype)
    out, kv = [], {}
    for i, l in enumerate(raw["layers"]):
        p, c = f"l{i}.", l["mixer"]
        h = token_shift(scalar_norm(x, t[p + "norm1"], eps), t[p + "shift"])
        j = c.get("kv_from")
        if j is None:
            kv[i] = keys_values(h, t, p + "mix.", c, eps)
        x = x + attention(h, t, p + "mix.", c, eps, kv[i if j is None else j])
        if l.get("mlp"):
            h = scalar_norm(x, t[p + "norm2"], eps)
            x = x + (dense_ff(h, t, p + "mlp.") if l["mlp"]["kind"] == "dense" else mixture(h, t, p + "mlp.", l["mlp"]))
        out.append(x)
    return torch.stack(out)


def forward(raw, t, ids, dtype=torch.float32):
    """Logits [T, vocab]."""
    x = scalar_norm(residuals(raw, t, ids, dtype)[-1], t["final.norm"], raw["norm"]["eps"])
    return matmul(x, t["head"]) * raw["logit_scale"]


# ---- random models --------------------------------------------------------------------------------------------------

def layer(heads, kv_heads, dim, vdim=None, size=0, scale=None, kv_from=None, mlp=None):
    c = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim or dim, "scale": dim ** -0.5 if scale is None else scale}
    if size:
        c["mask"] = {"size": size}
    if kv_from is not None:
        c["kv_from"] = kv_from
    return {"type": "attention", "mixer": c, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, identity=0, shared=0):
    r = {"experts": experts, "top": top}
    if identity:
        r["identity"] = identity
    return {"kind": "moe", "expert": {"ff": ff}, "router": r, **({"shared": {"ff": shared}} if shared else {})}


def config(layers, width, vocab=97, eps=1e-5, embed_scale=1.0, logit_scale=1.0, positions=1024):
    return {"architecture": "Pulunex", "embedding": {"scale": embed_scale}, "layers": layers, "logit_scale": logit_scale,
            "max_positions": positions, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def random_tensors(raw, seed=0):
    """Checkpoint tensors (bf16 values) of a configuration."""
    g = torch.Generator().manual_seed(seed)
    H, t = raw["width"], {}

    def put(name, *shape, k=1.0, shift=0.0):
        t[name] = (torch.randn(shape, generator=g) * k + shift).to(torch.bfloat16)

    def mat(name, n, k):
        put(name, n, k, k=k ** -0.5)

    def swiglu(p, ff):
        mat(p + "gate", ff, H), mat(p + "up", ff, H), mat(p + "down", H, ff)

    put("embed", raw["vocab"], H), put("pos", raw["max_positions"], H, k=0.5)
    for i, l in enumerate(raw["layers"]):
        p, c, f = f"l{i}.", l["mixer"], l.get("mlp")
        put(p + "norm1", k=0.2, shift=1.0), put(p + "shift", H, k=0.3, shift=0.4)
        m = p + "mix."
        rows = [("q", c["heads"] * c["dim"])] + ([] if "kv_from" in c else [("k", c["kv_heads"] * c["dim"]), ("v", c["kv_heads"] * c["vdim"])])
        for n, r in rows:
            mat(m + n, r, H), put(m + n + ".b", r, k=0.3)
        put(m + "talk", c["heads"], c["heads"], k=0.5)
        t[m + "talk"] = (t[m + "talk"].float() + torch.eye(c["heads"])).to(torch.bfloat16)
        mat(m + "o", H, c["heads"] * c["vdim"])
        if not f:
            continue
        put(p + "norm2", k=0.2, shift=1.0)
        m = p + "mlp."
        if f["kind"] == "dense":
            mat(m + "up", f["ff"], H), mat(m + "down", H, f["ff"])
            continue
        r = f["router"]
        for e in range(r["experts"]):
            swiglu(f"{m}e{e}.", f["expert"]["ff"])
        mat(m + "router", r["experts"] + r.get("identity", 0), H), put(m + "correction", r["experts"] + r.get("identity", 0), k=0.05)
        if f.get("shared"):
            swiglu(m + "shared.", f["shared"]["ff"]), mat(m + "shared.sg", 1, H)
    put("final.norm", k=0.2, shift=1.0), mat("head", raw["vocab"], H)
    return t
