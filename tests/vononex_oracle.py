"""Plain, slow definition of a Vononex decoder: whole sequences, fp32 (or fp64) torch, one function per mechanism, no cache and
no kernels.  The tests compare the framework with it; it shares no code with the package.

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


def norm(x, w, eps):
    return rms(x, eps) * w.to(x.dtype)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate(x, positions, dims, base, sign=1.0):
    """x [T, H, D]: values i and i + dims/2 of the first `dims` turn by position * base^(-2i/dims) (back with sign = -1)."""
    half = dims // 2
    f = float(base) ** (-2.0 * torch.arange(half, dtype=torch.float64) / dims)
    a = sign * (positions.to(torch.float64)[:, None] * f)[:, None, :]
    cos, sin = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], -1)


def causal_softmax(scores):
    """scores [H, T, S] of the last T of S positions."""
    T, S = scores.shape[-2:]
    mask = torch.arange(S)[None, :] <= torch.arange(S - T, S)[:, None]
    s = scores.masked_fill(~mask, float("-inf"))
    e = torch.exp(s - s.amax(-1, keepdim=True))
    return e / e.sum(-1, keepdim=True)


def turned_values(w, v, i, j, base):
    """sum_j w_ij v_j with v_j turned by its position j and the sum turned back by i: w [H, T, S], v [S, H, V]."""
    V = v.shape[-1]
    o = torch.einsum("hts,shv->thv", w, rotate(v, j, V, base))
    return rotate(o, i, V, base, -1.0)


def attention(h, t, p, c, eps):
    """Grouped-query attention: norm over the whole query / key rows, rotation, turned values, a temperature per head."""
    T, H, G, D, V = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    pos, rot = torch.arange(T), c["rot"]
    q, k, v = (matmul(h, t[p + n], t[p + n + ".b"]) for n in "qkv")
    q = rotate(norm(q, t[p + "q.norm"], eps).view(T, H, D), pos, rot["dims"], rot["base"])
    k = rotate(norm(k, t[p + "k.norm"], eps).view(T, G, D), pos, rot["dims"], rot["base"]).repeat_interleave(H // G, 1)
    s = torch.einsum("thd,shd->hts", q, k) * c["scale"] * t[p + "temp"].to(h.dtype)[:, None, None]
    o = turned_values(causal_softmax(s), v.view(T, G, V).repeat_interleave(H // G, 1), pos, pos, rot["base"])
    return matmul(o.reshape(T, H * V), t[p + "o"], t[p + "o.b"])


def retain(q, k, v, decay, S):
    """S <- decay S + k v^T, o = S^T q, token by token: q, k [T, H, D], v [T, H, V], decay [H], S [H, D, V]."""
    o = []
    for i in range(q.shape[0]):
        S = decay[:, None, None] * S + k[i][:, :, None] * v[i][:, None, :]
        o.append((S * q[i][:, :, None]).sum(1))
    return torch.stack(o), S


def retention(h, t, p, c, eps):
    T, H, D, V = h.shape[0], c["heads"], c["dim"], c["vdim"]
    pos, rot = torch.arange(T), c["rot"]
    q = rotate(matmul(h, t[p + "q"]).view(T, H, D), pos, rot["dims"], rot["base"])
    k = rotate(matmul(h, t[p + "k"]).view(T, H, D), pos, rot["dims"], rot["base"]) * D ** -0.5
    o, _ = retain(q, k, matmul(h, t[p + "v"]).view(T, H, V), torch.tensor(c["decay"], dtype=h.dtype), torch.zeros(H, D, V, dtype=h.dtype))
    return matmul(rms(o, eps).reshape(T, H * V) * silu(matmul(h, t[p + "g"])), t[p + "o"])


def parallel(h, t, p, c, eps):
    return c["left_scale"] * attention(h, t, p + "left.", c["left"], eps) + c["right_scale"] * retention(h, t, p + "right.", c["right"], eps)


def min_gru(z, u, S):
    """S <- (1 - z) S + z candidate(u): z, u [T, W], S [W].  Returns every token's S."""
    cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    out = []
    for i in range(z.shape[0]):
        S = (1 - z[i]) * S + z[i] * cand[i]
        out.append(S)
    return torch.stack(out)


def mingru(h, t, p, c, eps):
    z = torch.sigmoid(matmul(h, t[p + "z"], t[p + "z.b"]))
    S = min_gru(z, matmul(h, t[p + "x"], t[p + "x.b"]), torch.zeros(c["width"], dtype=h.dtype))
    return matmul(S * silu(matmul(h, t[p + "g"])), t[p + "o"])


def feed_forward(h, t, p):
    a = gelu_tanh(matmul(h, t[p + "gate"], t[p + "gate.b"])) * matmul(h, t[p + "up"], t[p + "up.b"])
    return matmul(a, t[p + "down"], t[p + "down.b"])


MIXERS = {"parallel": parallel, "mingru": mingru}


def residuals(raw, tensors, ids, dtype=torch.float32):
    """The residual stream after every layer, [layers, T, H]."""
    eps, alpha = raw["norm"]["eps"], raw["postln_alpha"]
    x = tensors["embed"].to(dtype)[torch.as_tensor(ids)]
    out = []
    for i, l in enumerate(raw["layers"]):
        p = f"l{i}."
        x = norm(alpha * x + MIXERS[l["type"]](x, tensors, p + "mix.", l["mixer"], eps), tensors[p + "norm1"], eps)
        if l.get("mlp") is not None:
            x = norm(alpha * x + feed_forward(x, tensors, p + "mlp."), tensors[p + "norm2"], eps)
        out.append(x)
    return torch.stack(out)


def forward(raw, tensors, ids, dtype=torch.float32):
    x = residuals(raw, tensors, ids, dtype)[-1]
    return matmul(norm(x, tensors["final.norm"], raw["norm"]["eps"]), tensors["head"])


# ---- random configurations and checkpoints ----------------------------------------------------------------------------

def dense(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def parallel_layer(heads=4, kv_heads=2, dim=16, vdim=16, dims=None, base=1e4, scale=None, left_scale=1.0, right_scale=1.0, r_heads=2,
                   r_dim=16, r_vdim=16, r_dims=None, r_base=1e5, decay=None, ff=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5,
            "rot": {"base": base, "dims": dims or dim}}
    right = {"heads": r_heads, "dim": r_dim, "vdim": r_vdim, "rot": {"base": r_base, "dims": r_dims or r_dim},
             "decay": decay or [1 - 2.0 ** (-3 - i) for i in range(r_heads)]}
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}, "mlp": dense(ff)}


def mingru_layer(width=32, ff=None):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": dense(ff)}


def config(layers, width=64, vocab=96, eps=1e-5, alpha=2.0):
    return {"architecture": "Vononex", "layers": layers, "norm": {"eps": eps}, "postln_alpha": alpha, "vocab": vocab, "width": width}


def random_tensors(raw, seed=0, dtype=torch.bfloat16):
    g = torch.Generator().manual_seed(seed)
    H = raw["width"]
    t = {}

    def mat(name, n, k, gain=1.0):
        t[name] = (torch.randn(n, k, generator=g) * gain * k ** -0.5).to(dtype)

    def vec(name, n, spread, shift=0.0):
        t[name] = (torch.randn(n, generator=g) * spread + shift).to(dtype)

    t["embed"] = torch.randn(raw["vocab"], H, generator=g).to(dtype)
    for i, l in enumerate(raw["layers"]):
        p, c = f"l{i}.", l["mixer"]
        vec(p + "norm1", H, 0.2, 1.0)
        m = p + "mix."
        if l["type"] == "mingru":
            W = c["width"]
            mat(m + "z", W, H), vec(m + "z.b", W, 1.0, -1.5), mat(m + "x", W, H, 2.0), vec(m + "x.b", W, 0.5), mat(m + "g", W, H), mat(m + "o", H, W, 2.0)
        else:
            a, r = c["left"], c["right"]
            for n, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                mat(m + "left." + n, rows, H), vec(m + "left." + n + ".b", rows, 0.5)
                if n != "v":
                    vec(m + "left." + n + ".norm", rows, 0.3, 1.0)
            vec(m + "left.temp", a["heads"], 0.3, 1.5)
            mat(m + "left.o", H, a["heads"] * a["vdim"], 2.0), vec(m + "left.o.b", H, 0.3)
            for n, rows in (("q", r["dim"]), ("k", r["dim"]), ("v", r["vdim"]), ("g", r["vdim"])):
                mat(m + "right." + n, r["heads"] * rows, H)
            mat(m + "right.o", H, r["heads"] * r["vdim"], 2.0)
        if l.get("mlp") is not None:
            f, p = l["mlp"]["ff"], p + "mlp."
            vec(f"l{i}.norm2", H, 0.2, 1.0)
            mat(p + "gate", f, H), vec(p + "gate.b", f, 0.5), mat(p + "up", f, H), vec(p + "up.b", f, 0.5), mat(p + "down", H, f, 2.0), vec(p + "down.b", H, 0.3)
    vec("final.norm", H, 0.2, 1.0)
    mat("head", raw["vocab"], H)
    return t
