"""Plain, slow definition of a Zemezen decoder: whole sequences, fp32 (or fp64) torch, one function per mechanism, no cache and
no kernels.  The tests compare the framework with it; it shares no code with the package.

Also makes small random configurations and checkpoints.
"""
import torch


# ---- mechanisms -----------------------------------------------------------------------------------------------------

def matmul(x, w):
    return x @ w.to(x.dtype).t()


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * w.to(x.dtype)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def rotate(x, positions, dims, base):
    """x [T, H, D]: values i and i + dims/2 of the first `dims` turn by position * base^(-2i/dims)."""
    half = dims // 2
    f = float(base) ** (-2.0 * torch.arange(half, dtype=torch.float64) / dims)
    a = (positions.to(torch.float64)[:, None] * f)[:, None, :]
    cos, sin = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], -1)


def visible(T, size=0, keep_first=0):
    """[query, key] mask: causal, the last `size` positions (0: all of them) and the first `keep_first`."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first)) if size else j <= i


def softmax_with_sink(scores, mask, sink=None):
    """scores [H, T, T], sink [H]: exp(sink) joins the denominator only."""
    s = scores.masked_fill(~mask, float("-inf"))
    top = s.amax(-1, keepdim=True)
    if sink is None:
        e = torch.exp(s - top)
        return e / e.sum(-1, keepdim=True)
    z = sink.to(s.dtype)[:, None, None]
    top = torch.maximum(top, z)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(z - top))


def attention(h, t, p, c, eps):
    """Grouped-query attention whose values are the key projections themselves."""
    T, H, G, D = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    pos = torch.arange(T)
    q = matmul(h, t[p + "q"]).view(T, H, D)
    v = matmul(h, t[p + "k"]).view(T, G, D)
    q = rotate(norm(q, t[p + "q.norm"], eps), pos, c["rot"]["dims"], c["rot"]["base"])
    k = rotate(norm(v, t[p + "k.norm"], eps), pos, c["rot"]["dims"], c["rot"]["base"])
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    mask = c.get("mask") or {}
    w = softmax_with_sink(torch.einsum("thd,shd->hts", q, k) * c["scale"], visible(T, mask.get("size", 0), mask.get("keep_first", 0)), t[p + "sink"])
    return matmul(torch.einsum("hts,shd->thd", w, v).reshape(T, H * D), t[p + "o"])


def latent_attention(h, t, p, c, eps):
    T, H = h.shape[0], c["heads"]
    q = matmul(h, t[p + "q"]).view(T, H, c["dim"])
    lat = norm(matmul(h, t[p + "dkv"]), t[p + "dkv.norm"], eps)
    k = matmul(lat, t[p + "uk"]).view(T, H, c["dim"])
    v = matmul(lat, t[p + "uv"]).view(T, H, c["vdim"])
    w = softmax_with_sink(torch.einsum("thd,shd->hts", q, k) * c["scale"], visible(T))
    return matmul(torch.einsum("hts,shd->thd", w, v).reshape(T, H * c["vdim"]), t[p + "o"])


def short_conv(x, w):
    """Causal convolution per channel, x [T, C], w [C, taps]; then silu."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return silu(sum(padded[j:j + x.shape[0]] * w[:, j].to(x.dtype) for j in range(taps)))


def channel_decay(h, t, p, heads, dim):
    z = matmul(matmul(h, t[p + "a1"]), t[p + "a2"]) + t[p + "dt_bias"].to(h.dtype)
    rate = torch.exp(t[p + "A_log"].to(h.dtype))[None, :, None]
    return torch.exp(-rate * softplus(z).view(-1, heads, dim))


def delta_recurrence(q, k, v, g, beta):
    """q, k, g [T, H, dk], v [T, H, dv], beta [T, H]."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[-1], dtype=q.dtype)
    o = torch.empty(T, H, v.shape[-1], dtype=q.dtype)
    for i in range(T):
        S = g[i][:, :, None] * S
        u = beta[i][:, None] * (v[i] - (S * k[i][:, :, None]).sum(1))
        S = S + k[i][:, :, None] * u[:, None, :]
        o[i] = (S * q[i][:, :, None]).sum(1)
    return o


def channel_delta(h, t, p, c, eps):
    T, H, G, dk, dv = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (short_conv(matmul(h, t[p + n]), t[p + n + ".conv"]) for n in "qkv")
    q = (unit(q.view(T, G, dk)) * dk ** -0.5).repeat_interleave(H // G, 1)
    k = unit(k.view(T, G, dk)).repeat_interleave(H // G, 1)
    beta = torch.sigmoid(matmul(h, t[p + "b"]))
    o = delta_recurrence(q, k, v.view(T, H, dv), channel_decay(h, t, p, H, dk), beta)
    gate = torch.sigmoid(matmul(matmul(h, t[p + "g1"]), t[p + "g2"]))
    return matmul(norm(o, t[p + "norm"], eps).reshape(T, H * dv) * gate, t[p + "o"])


def feed_forward(h, t, p):
    return matmul(silu(matmul(h, t[p + "gate"])) * matmul(h, t[p + "up"]), t[p + "down"])


def choose_experts(z, top, groups=1, keep=1):
    """Logits z [T, E] -> weights [T, E], zero outside each row's choice: the best `keep` of `groups` runs of neighbours (by
    their largest score), then the `top` largest scores in them."""
    s = torch.softmax(z, -1)
    T, E = s.shape
    by_group = s.view(T, groups, E // groups).amax(-1)
    kept = torch.zeros(T, groups, dtype=torch.bool).scatter_(1, by_group.topk(keep, -1).indices, True)
    allowed = kept.repeat_interleave(E // groups, 1)
    chosen = s.masked_fill(~allowed, -1.0).topk(top, -1).indices
    return torch.zeros_like(s).scatter(1, chosen, s.gather(1, chosen))


def experts(h, t, p, c):
    r = c["router"]
    gr = r.get("groups") or {"count": 1, "keep": 1}
    w = choose_experts(matmul(h, t[p + "router"]), r["top"], gr["count"], gr["keep"])
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        rows = w[:, e].nonzero().squeeze(1)
        if rows.numel():
            out[rows] += w[rows, e, None] * feed_forward(h[rows], t, f"{p}e{e}.")
    return out


MIXERS = {"attention": attention, "latent_attention": latent_attention, "channel_delta": channel_delta}


def forward(raw, t, ids, dtype=torch.float32, trace=None):
    """Logits [T, vocab] of one sequence; `trace` (a list) collects the residual stream after every layer."""
    eps = raw["norm"]["eps"]
    x = t["embed"][torch.as_tensor(ids)].to(dtype)
    for i, layer in enumerate(raw["layers"]):
        p = f"l{layer.get('weights_of', i)}."
        h = norm(x, t[p + "norm1"], eps)
        y = MIXERS[layer["type"]](h, t, p + "mix.", layer["mixer"], eps)
        mlp = layer.get("mlp")
        if mlp:
            y = y + (feed_forward(h, t, p + "mlp.") if mlp["kind"] == "dense" else experts(h, t, p + "mlp.", mlp))
        x = x + y
        if trace is not None:
            trace.append(x)
    return matmul(norm(x, t["final.norm"], eps), t["head"])


# ---- small random models --------------------------------------------------------------------------------------------

def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(count, top, ff, groups=None, keep=None):
    r = {"experts": count, "top": top}
    if groups:
        r["groups"] = {"count": groups, "keep": keep}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def attention_layer(heads=4, kv_heads=2, dim=16, dims=None, base=10000.0, window=9, keep=2, scale=None, mlp=None):
    return _layer("attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "rot": {"base": base, "dims": dims or dim},
                                "mask": {"size": window, "keep_first": keep} if window else None,
                                "scale": scale if scale is not None else dim ** -0.5}, mlp)


def latent_layer(heads=3, dim=16, vdim=24, kv_rank=40, scale=None, mlp=None):
    return _layer("latent_attention", {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank,
                                       "scale": scale if scale is not None else dim ** -0.5}, mlp)


def delta_layer(heads=4, kv_heads=2, dim=16, vdim=24, conv=4, mlp=None):
    return _layer("channel_delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, mlp)


def config(layers, width=48, vocab=97, eps=1e-5):
    """A layer given as a number uses that layer's weights."""
    out = [dict(layers[l], weights_of=l) if isinstance(l, int) else l for l in layers]
    return {"architecture": "Zemezen", "layers": out, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def random_tensors(raw, seed=0, ranks=(6, 5)):
    """bf16 checkpoint tensors of a configuration; `ranks`: widths of the low-rank decay and gate.  Norm weights, biases and sinks
    are spread so that leaving one out or mixing two up shows in the logits."""
    g = torch.Generator().manual_seed(seed)
    W, V = raw["width"], raw["vocab"]

    def mat(n, k, gain=1.0):
        return (torch.randn(n, k, generator=g) * gain * k ** -0.5).to(torch.bfloat16)

    def vec(n, spread, shift=0.0):
        return (torch.randn(n, generator=g) * spread + shift).to(torch.bfloat16)

    t = {"embed": torch.randn(V, W, generator=g).to(torch.bfloat16), "final.norm": vec(W, 0.3, 1.0), "head": mat(V, W)}

    def feed(p, ff):
        t[p + "gate"], t[p + "up"], t[p + "down"] = mat(ff, W), mat(ff, W), mat(W, ff)

    for i, layer in enumerate(raw["layers"]):
        if "weights_of" in layer:
            continue
        p, c, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        t[p + "norm1"] = vec(W, 0.3, 1.0)
        if mlp and mlp["kind"] == "dense":
            feed(p + "mlp.", mlp["ff"])
        elif mlp:
            for e in range(mlp["router"]["experts"]):
                feed(f"{p}mlp.e{e}.", mlp["expert"]["ff"])
            t[p + "mlp.router"] = mat(mlp["router"]["experts"], W, 3.0)
        p, H, D = p + "mix.", c["heads"], c["dim"]
        if layer["type"] == "attention":
            t[p + "q"], t[p + "k"], t[p + "o"] = mat(H * D, W), mat(c["kv_heads"] * D, W), mat(W, H * D)
            t[p + "q.norm"], t[p + "k.norm"], t[p + "sink"] = vec(D, 0.4, 1.5), vec(D, 0.4, 1.5), vec(H, 1.0, 1.0)
        elif layer["type"] == "latent_attention":
            R = c["kv_rank"]
            t[p + "q"], t[p + "dkv"], t[p + "dkv.norm"] = mat(H * D, W, 2.0), mat(R, W), vec(R, 0.3, 1.0)
            t[p + "uk"], t[p + "uv"], t[p + "o"] = mat(H * D, R), mat(H * c["vdim"], R), mat(W, H * c["vdim"])
        else:
            for n, rows in (("q", c["kv_heads"] * D), ("k", c["kv_heads"] * D), ("v", H * c["vdim"])):
                t[p + n], t[p + n + ".conv"] = mat(rows, W), mat(rows, c["conv"], 1.5)
            t[p + "b"], t[p + "A_log"], t[p + "norm"] = mat(H, W), vec(H, 0.7, 0.5), vec(c["vdim"], 0.3, 1.0)
            t[p + "a1"], t[p + "a2"], t[p + "dt_bias"] = mat(ranks[0], W), mat(H * D, ranks[0]), vec(H * D, 1.5, -3.0)
            t[p + "g1"], t[p + "g2"], t[p + "o"] = mat(ranks[1], W), mat(H * c["vdim"], ranks[1], 2.0), mat(W, H * c["vdim"])
    return t
