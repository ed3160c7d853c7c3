"""Plain restatement of the Fiferax decoder in float64, one function per mechanism (test infrastructure, never on the
product path).  Every function takes whole sequences and loops over tokens where the mathematics is a recurrence; nothing
is cached, fused or chunked.  ``forward`` takes the parsed config.json and a name -> tensor mapping and returns the
logits of every position; ``make_config`` / ``make_weights`` draw small random models for the tests.

Mechanism functions return float64 tensors; ``x`` is [tokens, width] of one sequence.
"""
import math

import torch

F64 = torch.float64


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def rotary_half(x, pos, dims, base):
    """x [tokens, heads, dim]: the first ``dims`` dimensions rotated, i paired with i + dims / 2."""
    out = x.clone()
    h = dims // 2
    for i in range(h):
        a = pos.to(F64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, i], x[:, :, i + h]
        out[:, :, i] = u * c - v * s
        out[:, :, i + h] = v * c + u * s
    return out


def window_attention(q, k, v, scale, window):
    """q [T, H, D], k [T, G, D], v [T, G, Dv]; query i sees keys i - window + 1 .. i.  Returns [T, H, Dv]."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for i in range(T):
        lo = max(0, i - window + 1)
        for h in range(H):
            s = (k[lo:i + 1, h // per] @ q[i, h]) * scale
            p = torch.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[lo:i + 1, h // per]
    return out


def window_attention_fast(q, k, v, scale, window):
    """The same with the loops over i and h turned into one masked product (long test sequences)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    kk, vv = k.repeat_interleave(per, 1), v.repeat_interleave(per, 1)
    s = torch.einsum("ihd,jhd->hij", q, kk) * scale
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    s = s.masked_fill(((d < 0) | (d >= window))[None], -math.inf)
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), vv)


def delta_recurrence(r, k, v, w, a, state=None):
    """r, k, w, a [T, H, D] (w decay, a removal rate), v [T, H, Dv]: S <- diag(w) S - (a u)(u^T S) + k v^T with the unit
    key u and both terms on the old S; o = S^T r.  Returns (o [T, H, Dv], final S [H, D, Dv])."""
    T, H, D = k.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=F64) if state is None else state
    o = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for t in range(T):
        u = k[t] / torch.sqrt((k[t] * k[t]).sum(-1, keepdim=True) + 1e-6)
        seen = torch.einsum("hd,hde->he", u, S)
        S = w[t][:, :, None] * S - (a[t] * u)[:, :, None] * seen[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hde,hd->he", S, r[t])
    return o, S


def decay_recurrence(q, k, v, decay, state=None):
    """S <- decay_h S + k v^T, o = S^T q.  q, k [T, H, D], v [T, H, Dv], decay [H]."""
    T, H, D = k.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=F64) if state is None else state
    o = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hde,hd->he", S, q[t])
    return o, S


def min_gru(z, u, state=None):
    """z, u [T, W] before their non-linearities: S <- (1 - sigmoid(z)) S + sigmoid(z) g(u), g(u) = u + 1/2 for u >= 0 and
    sigmoid(u) below.  Returns (S of every step [T, W], final S)."""
    S = torch.zeros(z.shape[1], dtype=F64) if state is None else state
    out = torch.zeros_like(z)
    for t in range(z.shape[0]):
        g = sigmoid(z[t])
        cand = torch.where(u[t] >= 0, u[t] + 0.5, sigmoid(u[t]))
        S = (1.0 - g) * S + g * cand
        out[t] = S
    return out, S


def general_delta_mixer(h, W, p, m, eps):
    H, D = m["heads"], m["dim"]
    T = h.shape[0]
    lin = lambda n: h @ W(p + n).T  # noqa: E731
    heads = lambda x: x.view(T, H, -1)  # noqa: E731
    w = torch.exp(-math.exp(-0.5) * sigmoid(torch.tanh(lin("w1")) @ W(p + "w2").T + W(p + "w0")))
    a = sigmoid(lin("a") + W(p + "a.b"))
    o, _ = delta_recurrence(heads(lin("r")), heads(lin("k")), heads(lin("v")), heads(w), heads(a))
    o = rms_norm(o, 1.0, eps).reshape(T, -1) * W(p + "norm")
    return (o * sigmoid(lin("g"))) @ W(p + "o").T


def attention_mixer(h, W, p, m, eps, fast=True):
    T, D = h.shape[0], m["dim"]
    q = (h @ W(p + "q").T).view(T, m["heads"], D)
    k = (h @ W(p + "k").T).view(T, m["kv_heads"], D)
    v = k
    pos = torch.arange(T)
    q = rotary_half(rms_norm(q, W(p + "q.norm"), eps), pos, m["rot"]["dims"], m["rot"]["base"])
    k = rotary_half(rms_norm(k, W(p + "k.norm"), eps), pos, m["rot"]["dims"], m["rot"]["base"])
    o = (window_attention_fast if fast else window_attention)(q, k, v, m["scale"], m["mask"]["size"])
    return o.reshape(T, -1) @ W(p + "o").T


def lightning_mixer(h, W, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q, k, v = (silu(h @ W(p + n).T).view(T, H, -1) for n in "qkv")
    o, _ = decay_recurrence(q, k, v, torch.tensor(m["decay"], dtype=F64))
    o = rms_norm(o.reshape(T, -1), W(p + "norm"), eps)
    return (o * sigmoid(h @ W(p + "g").T)) @ W(p + "o").T


def parallel_mixer(h, W, p, m, eps):
    return m["left_scale"] * attention_mixer(h, W, p + "left.", m["left"], eps) + \
        m["right_scale"] * lightning_mixer(h, W, p + "right.", m["right"], eps)


def min_gru_mixer(h, W, p, m, eps):
    S, _ = min_gru(h @ W(p + "z").T + W(p + "z.b"), h @ W(p + "x").T + W(p + "x.b"))
    return (S * silu(h @ W(p + "g").T)) @ W(p + "o").T


MIXERS = {"general_delta": general_delta_mixer, "parallel": parallel_mixer, "mingru": min_gru_mixer}


def mlp(h, W, p):
    return (gelu_tanh(h @ W(p + "gate").T) * (h @ W(p + "up").T)) @ W(p + "down").T


def forward(config, tensors, tokens, want_layers=False):
    """Logits [T, vocab] of one sequence (and the residual stream after every layer [L, T, width])."""
    cache = {}

    def W(name):
        if name not in cache:
            cache[name] = tensors[name].to(F64)
        return cache[name]

    eps = config["norm"]["eps"]
    x = W("embed")[torch.as_tensor(tokens)] * config["embedding"]["scale"]
    layers = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        x = x + MIXERS[layer["type"]](rms_norm(x, W(p + "norm1"), eps), W, p + "mix.", layer["mixer"], eps)
        if layer["mlp"] is not None:
            x = x + mlp(rms_norm(x, W(p + "norm2"), eps), W, p + "mlp.")
        layers.append(x)
    logits = rms_norm(x, W("final.norm"), eps) @ W("head").T
    return (logits, torch.stack(layers)) if want_layers else logits


# ---------------------------------------------------------------------------------------------- small random models
def make_config(width, vocab, layers, eps=1e-5, scale=2.0):
    return {"architecture": "Fiferax", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps},
            "vocab": vocab, "width": width}


def delta_layer(heads, dim, ff=None):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}, "mlp": dense(ff)}


def gru_layer(width, ff=None):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": dense(ff)}


def parallel_layer(heads, kv_heads, dim, window, rot_dims, base, scale, r_heads, r_dim, r_vdim, decay, left_scale=1.0,
                   right_scale=1.0, ff=None):
    return {"type": "parallel", "mlp": dense(ff), "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": window},
                 "rot": {"dims": rot_dims, "base": base}, "scale": scale},
        "right": {"heads": r_heads, "dim": r_dim, "vdim": r_vdim, "decay": list(decay)},
        "left_scale": left_scale, "right_scale": right_scale}}


def dense(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def tensor_shapes(config, rank=8):
    """name -> shape of every tensor the design has for this configuration; ``rank``: rows of the decay's first factor."""
    d = config["width"]
    s = {"embed": (config["vocab"], d), "final.norm": (d,), "head": (config["vocab"], d)}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        s[p + "norm1"] = (d,)
        if layer["type"] == "general_delta":
            n = m["heads"] * m["dim"]
            for name in "rkvga":
                s[p + "mix." + name] = (n, d)
            s.update({p + "mix.a.b": (n,), p + "mix.w1": (rank, d), p + "mix.w2": (n, rank), p + "mix.w0": (n,),
                      p + "mix.norm": (n,), p + "mix.o": (d, n)})
        elif layer["type"] == "mingru":
            n = m["width"]
            for name in "zxg":
                s[p + "mix." + name] = (n, d)
            s.update({p + "mix.z.b": (n,), p + "mix.x.b": (n,), p + "mix.o": (d, n)})
        else:
            L, R = m["left"], m["right"]
            s.update({p + "mix.left.q": (L["heads"] * L["dim"], d), p + "mix.left.k": (L["kv_heads"] * L["dim"], d),
                      p + "mix.left.q.norm": (L["dim"],), p + "mix.left.k.norm": (L["dim"],),
                      p + "mix.left.o": (d, L["heads"] * L["dim"])})
            n, nv = R["heads"] * R["dim"], R["heads"] * R["vdim"]
            s.update({p + "mix.right.q": (n, d), p + "mix.right.k": (n, d), p + "mix.right.v": (nv, d),
                      p + "mix.right.g": (nv, d), p + "mix.right.norm": (nv,), p + "mix.right.o": (d, nv)})
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            s.update({p + "norm2": (d,), p + "mlp.gate": (ff, d), p + "mlp.up": (ff, d), p + "mlp.down": (d, ff)})
    return s


def make_weights(config, seed, rank=8):
    """Seeded random bf16 tensors: rows of unit gain, norms around 1, biases spread over +-1."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in sorted(tensor_shapes(config, rank).items()):
        t = torch.randn(*shape, generator=g)
        if len(shape) == 2:
            t = t * (1.0 if name == "embed" else shape[1] ** -0.5)
        elif "norm" in name:
            t = 1.0 + 0.2 * t
        out[name] = t.to(torch.bfloat16)
    return out
