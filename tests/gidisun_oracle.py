"""Plain, slow definition of a Gidisun decoder: whole sequences, fp32 (or fp64) torch, one function per mechanism,
no cache and no kernels.  The tests compare the framework with it; it shares no code with the package.

Also makes small random configurations and checkpoints.
"""
import math

import torch


# ---- mechanisms -----------------------------------------------------------------------------------------------------

def matmul(x, w):
    return x @ w.to(x.dtype).t()


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_zero(x, w, eps):
    return rms(x, eps) * (1.0 + w.to(x.dtype))


def silu(z):
    return z * torch.sigmoid(z)


def yarn_frequencies(dims, base, scaling):
    """(rotation frequency of every pair, factor on cos and sin) as fp64."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = float(base) ** (-2.0 * i / dims)
    if not scaling:
        return f, 1.0

    def dim_of(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(dim_of(scaling["fast"])), 0)
    hi = min(math.ceil(dim_of(scaling["slow"])), dims - 1)
    ramp = torch.clamp((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / scaling["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_half(x, positions, rot):
    """x [T, ..., D]: pair (i, i + dims/2) of the first `dims` values turned by position * f_i; the rest pass."""
    dims = rot["dims"]
    f, m = yarn_frequencies(dims, rot["base"], rot.get("scaling"))
    a = positions.to(torch.float64)[:, None] * f[None, :]
    cos, sin = (torch.cos(a) * m).to(x.dtype), (torch.sin(a) * m).to(x.dtype)
    while cos.dim() < x.dim():
        cos, sin = cos.unsqueeze(1), sin.unsqueeze(1)
    u, v, rest = x[..., :dims // 2], x[..., dims // 2:dims], x[..., dims:]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, rest], -1)


def window_mask(T, size):
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) if not size else ((d >= 0) & (d < size))


def sink_softmax(scores, mask, sink):
    """Softmax over the keys a query sees with exp(sink) added to the denominator.  scores [H, T, T], sink [H]."""
    s = scores.masked_fill(~mask, float("-inf"))
    s0 = sink.to(s.dtype)[:, None, None]
    top = torch.maximum(s.amax(-1, keepdim=True), s0)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(s0 - top))


def latent_attention(h, t, p, c, eps):
    T, H = h.shape[0], c["heads"]
    pos = torch.arange(T)
    q = matmul(h, t[p + "q"]).view(T, H, c["dim"] + c["rot_dim"])
    q_plain, q_rot = q[..., :c["dim"]], rotate_half(q[..., c["dim"]:], pos, c["rot"])
    d = matmul(h, t[p + "dkv"])
    lat = rms(d[:, :c["kv_rank"]], eps) * t[p + "dkv.norm"].to(h.dtype)
    k_rot = rotate_half(d[:, c["kv_rank"]:], pos, c["rot"])
    k_plain = matmul(lat, t[p + "uk"]).view(T, H, c["dim"])
    v = matmul(lat, t[p + "uv"]).view(T, H, c["vdim"])
    s = (torch.einsum("thd,shd->hts", q_plain, k_plain) + torch.einsum("thd,sd->hts", q_rot, k_rot)) * c["scale"]
    w = sink_softmax(s, window_mask(T, (c.get("mask") or {}).get("size")), t[p + "sink"])
    o = torch.einsum("hts,shd->thd", w, v).reshape(T, H * c["vdim"])
    return matmul(o, t[p + "o"])


def gla_decay(h, t, p, c):
    z = matmul(matmul(h, t[p + "a1"]), t[p + "a2"]) + t[p + "a2.b"].to(h.dtype)
    return torch.sigmoid(z).pow(1.0 / c["tau"]).view(-1, c["heads"], c["dim"])


def gla_recurrence(q, k, v, alpha):
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[-1], dtype=q.dtype)
    o = torch.empty(T, H, v.shape[-1], dtype=q.dtype)
    for i in range(T):
        S = alpha[i][:, :, None] * S + k[i][:, :, None] * v[i][:, None, :]
        o[i] = (S * q[i][:, :, None]).sum(1)
    return o


def gla(h, t, p, c, eps):
    T, H = h.shape[0], c["heads"]
    q = matmul(h, t[p + "q"]).view(T, H, c["dim"]) * c["dim"] ** -0.5
    k = matmul(h, t[p + "k"]).view(T, H, c["dim"])
    v = matmul(h, t[p + "v"]).view(T, H, c["vdim"])
    o = rms(gla_recurrence(q, k, v, gla_decay(h, t, p, c)), eps) * t[p + "norm"].to(h.dtype)
    o = o.reshape(T, H * c["vdim"]) * silu(matmul(h, t[p + "g"]))
    return matmul(o, t[p + "o"])


def mlstm_gates(h, t, p, c):
    cap = c["gate_cap"]
    i = cap * torch.tanh((matmul(h, t[p + "i"]) + t[p + "i.b"].to(h.dtype)) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((matmul(h, t[p + "f"]) + t[p + "f.b"].to(h.dtype)) / cap))
    return i, f


def mlstm_recurrence(q, k, v, i, f):
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[-1], dtype=q.dtype)
    n = torch.zeros(H, dk, dtype=q.dtype)
    m = torch.zeros(H, dtype=q.dtype)
    o = torch.empty(T, H, v.shape[-1], dtype=q.dtype)
    for s in range(T):
        m_new = torch.maximum(f[s] + m, i[s])
        keep, add = torch.exp(f[s] + m - m_new), torch.exp(i[s] - m_new)
        S = keep[:, None, None] * S + add[:, None, None] * k[s][:, :, None] * v[s][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[s]
        m = m_new
        den = torch.maximum((n * q[s]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        o[s] = (S * q[s][:, :, None]).sum(1) / den[:, None]
    return o


def mlstm(h, t, p, c, eps):
    T, H = h.shape[0], c["heads"]
    q = matmul(h, t[p + "q"]).view(T, H, c["dim"]) * c["dim"] ** -0.5
    k = matmul(h, t[p + "k"]).view(T, H, c["dim"])
    v = matmul(h, t[p + "v"]).view(T, H, c["vdim"])
    i, f = mlstm_gates(h, t, p, c)
    o = rms(mlstm_recurrence(q, k, v, i, f), eps).reshape(T, H * c["vdim"])
    o = o * t[p + "norm"].to(h.dtype) * torch.sigmoid(matmul(h, t[p + "g"]))
    return matmul(o, t[p + "o"])


def feed_forward(h, t, p):
    return matmul(silu(matmul(h, t[p + "gate"])) * matmul(h, t[p + "up"]), t[p + "down"])


MIXERS = {"latent_attention": latent_attention, "gla": gla, "mlstm": mlstm}


def forward(raw, t, ids, dtype=torch.float32, trace=None):
    """Logits [T, vocab] of one sequence; `trace` (a list) collects the residual stream after every layer."""
    eps = raw["norm"]["eps"]
    x = t["embed"][torch.as_tensor(ids)].to(dtype)
    for i, layer in enumerate(raw["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](norm_around_zero(x, t[p + "norm1"], eps), t, p + "mix.", layer["mixer"], eps)
        x = x + norm_around_zero(y, t[p + "norm1b"], eps)
        if layer.get("mlp"):
            y = feed_forward(norm_around_zero(x, t[p + "norm2"], eps), t, p + "mlp.")
            x = x + norm_around_zero(y, t[p + "norm2b"], eps)
        if trace is not None:
            trace.append(x)
    return matmul(norm_around_zero(x, t["final.norm"], eps), t["head"])


# ---- small random models --------------------------------------------------------------------------------------------

def attention_layer(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=40, window=9, base=10000.0, scaling=None, scale=None, dims=None,
                    ff=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
             "mask": {"size": window} if window else None, "rot": {"base": base, "dims": dims or rot_dim, "scaling": scaling},
             "scale": scale if scale is not None else (dim + rot_dim) ** -0.5}
    return {"type": "latent_attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def gla_layer(heads=2, dim=16, vdim=24, tau=8.0, ff=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def mlstm_layer(heads=2, dim=24, vdim=16, cap=15.0, ff=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=48, vocab=97, eps=1e-5):
    return {"architecture": "Gidisun", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def random_tensors(raw, seed=0, low_rank=8):
    """bf16 checkpoint tensors of a configuration.  Norm weights, biases and sinks are spread so that leaving one out or
    mixing two up shows in the logits."""
    g = torch.Generator().manual_seed(seed)
    W, V = raw["width"], raw["vocab"]

    def mat(n, k, gain=1.0):
        return (torch.randn(n, k, generator=g) * gain * k ** -0.5).to(torch.bfloat16)

    def vec(n, spread, shift=0.0):
        return (torch.randn(n, generator=g) * spread + shift).to(torch.bfloat16)

    t = {"embed": (torch.randn(V, W, generator=g)).to(torch.bfloat16), "final.norm": vec(W, 0.3), "head": mat(V, W)}
    for i, layer in enumerate(raw["layers"]):
        p, c = f"l{i}.", layer["mixer"]
        t[p + "norm1"], t[p + "norm1b"] = vec(W, 0.3), vec(W, 0.3)
        if layer.get("mlp"):
            ff = layer["mlp"]["ff"]
            t[p + "norm2"], t[p + "norm2b"] = vec(W, 0.3), vec(W, 0.3)
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = mat(ff, W), mat(ff, W), mat(W, ff)
        p, H = p + "mix.", c["heads"]
        if layer["type"] == "latent_attention":
            R = c["kv_rank"]
            t[p + "q"] = mat(H * (c["dim"] + c["rot_dim"]), W, 2.0)
            t[p + "dkv"], t[p + "dkv.norm"] = mat(R + c["rot_dim"], W), vec(R, 0.3, 1.0)
            t[p + "uk"], t[p + "uv"] = mat(H * c["dim"], R), mat(H * c["vdim"], R)
            t[p + "sink"], t[p + "o"] = vec(H, 1.0, 1.0), mat(W, H * c["vdim"])
            continue
        for n, d in (("q", c["dim"]), ("k", c["dim"]), ("v", c["vdim"]), ("g", c["vdim"])):
            t[p + n] = mat(H * d, W)
        t[p + "o"] = mat(W, H * c["vdim"])
        if layer["type"] == "gla":
            t[p + "norm"] = vec(c["vdim"], 0.3, 1.0)
            t[p + "a1"], t[p + "a2"], t[p + "a2.b"] = mat(low_rank, W), mat(H * c["dim"], low_rank), vec(H * c["dim"], 2.0, 1.0)
        else:
            t[p + "norm"] = vec(H * c["vdim"], 0.3, 1.0)
            t[p + "i"], t[p + "i.b"] = mat(H, W), vec(H, 1.0, -1.0)
            t[p + "f"], t[p + "f.b"] = mat(H, W), vec(H, 1.0, 3.0)
    return t
