"""Plain restatement of the Molitar decoder in float64, one function per mechanism (test infrastructure, never on the
product path).  Every function takes whole sequences; nothing is cached, fused, absorbed or chunked.  ``forward`` takes the
parsed config.json and a name -> tensor mapping and returns the logits of every position; ``make_config`` /
``make_weights`` draw small random models for the tests.

Mechanism functions return float64 tensors; ``x`` is [tokens, width] of one sequence.
"""
import math

import torch

F64 = torch.float64


def rms(x, eps):
    """x over the root of its mean square, eps inside the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def offset_norm(x, w, eps):
    """RMS norm whose stored weight is the difference from one."""
    return rms(x, eps) * (1.0 + w)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def rotation_frequencies(dims, base, scaling=None):
    """Angle per position of every pair, and the factor on cos and sin.  With YaRN scaling, pairs that turn more than
    ``fast`` times within the original context keep their frequency, those below ``slow`` turns are slowed by ``factor``,
    with a linear ramp over the pair index in between."""
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return freq, 1.0

    def pair_of(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    first = max(math.floor(pair_of(scaling["fast"])), 0)
    last = min(math.ceil(pair_of(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        r = min(max((i - first) / max(last - first, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * r + f * (1.0 - r))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotary_pairs(x, pos, dims, base, scaling=None):
    """x [tokens, heads, dim]: neighbours (2 i, 2 i + 1) of the first ``dims`` dimensions rotated by position * frequency."""
    freq, amp = rotation_frequencies(dims, base, scaling)
    out = x.clone()
    for i, f in enumerate(freq):
        a = pos.to(F64) * f
        c, s = (amp * torch.cos(a))[:, None], (amp * torch.sin(a))[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * c - v * s
        out[:, :, 2 * i + 1] = v * c + u * s
    return out


def causal_attention(q, k, v, scale, softcap=None, sink=None):
    """q [T, H, D], k [T, G, D], v [T, G, Dv], one query and head at a time: capped scores of keys 0 .. i, softmax whose
    denominator also counts exp(sink of the head).  Returns [T, H, Dv]."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for i in range(T):
        for h in range(H):
            s = (k[:i + 1, h // per] @ q[i, h]) * scale
            if softcap is not None:
                s = softcap * torch.tanh(s / softcap)
            top = s.max() if sink is None else torch.maximum(s.max(), sink[h])
            p = torch.exp(s - top)
            total = p.sum() if sink is None else p.sum() + torch.exp(sink[h] - top)
            out[i, h] = (p / total) @ v[:i + 1, h // per]
    return out


def causal_attention_fast(q, k, v, scale, softcap=None, sink=None):
    """The same as one masked product, the sink as a column of scores without a value (long test sequences)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    kk, vv = k.repeat_interleave(per, 1), v.repeat_interleave(per, 1)
    s = torch.einsum("ihd,jhd->hij", q, kk) * scale
    if softcap is not None:
        s = softcap * torch.tanh(s / softcap)
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), -math.inf)
    if sink is None:
        return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), vv)
    p = torch.softmax(torch.cat([s, sink[:, None, None].expand(H, T, 1)], -1), -1)
    return torch.einsum("hij,jhd->ihd", p[..., :T], vv)


def mix_values(v, first, lam):
    return (1.0 - lam) * v + lam * first


def attention_mixer(h, W, p, m, eps, shared, fast=True):
    """``shared``: the values of the first layer that mixes values, filled in by that layer."""
    T = h.shape[0]

    def lin(n, size):
        return (h @ W(p + n).T + W(p + n + ".b")).view(T, -1, size)

    q, k, v = lin("q", m["dim"]), lin("k", m["dim"]), lin("v", m["vdim"])
    pos = torch.arange(T)
    rot = m["rot"]
    q = rotary_pairs(q, pos, rot["dims"], rot["base"], rot.get("scaling"))
    k = rotary_pairs(k, pos, rot["dims"], rot["base"], rot.get("scaling"))
    if m.get("v_mix"):
        if "v" in shared:
            v = mix_values(v, shared["v"], W(p + "vmix"))
        else:
            shared["v"] = v
    attend = causal_attention_fast if fast else causal_attention
    o = attend(q, k, v, m["scale"], m["softcap"], W(p + "sink")).reshape(T, -1)
    return (o * sigmoid(h @ W(p + "g").T)) @ W(p + "o").T


def latent_attention_mixer(h, W, p, m, eps, shared, fast=True):
    T, H, D, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    rot = m["rot"]
    pos = torch.arange(T)
    c_q = rms(h @ W(p + "dq").T, eps) * W(p + "dq.norm")
    q = (c_q @ W(p + "uq").T).view(T, H, D + R)
    down = h @ W(p + "dkv").T
    c = rms(down[:, :m["kv_rank"]], eps) * W(p + "dkv.norm")
    turn = lambda t: rotary_pairs(t, pos, rot["dims"], rot["base"], rot.get("scaling"))  # noqa: E731
    shared_key = turn(down[:, None, m["kv_rank"]:])
    q = torch.cat([q[..., :D], turn(q[..., D:])], -1)
    k = torch.cat([(c @ W(p + "uk").T).view(T, H, D), shared_key.expand(T, H, R)], -1)
    v = (c @ W(p + "uv").T).view(T, H, m["vdim"])
    o = (causal_attention_fast if fast else causal_attention)(q, k, v, m["scale"])
    return o.reshape(T, -1) @ W(p + "o").T


MIXERS = {"attention": attention_mixer, "latent_attention": latent_attention_mixer}


def mlp(h, W, p):
    return (silu(h @ W(p + "gate").T) * (h @ W(p + "up").T)) @ W(p + "down").T


def forward(config, tensors, tokens, want_layers=False):
    """Logits [T, vocab] of one sequence (and the residual stream after every layer [L, T, width])."""
    cache = {}

    def W(name):
        if name not in cache:
            cache[name] = tensors[name].to(F64)
        return cache[name]

    eps, m = config["norm"]["eps"], config["residual_mult"]
    x = W("embed")[torch.as_tensor(tokens)]
    layers, shared = [], {}
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](offset_norm(x, W(p + "norm1"), eps), W, p + "mix.", layer["mixer"], eps, shared)
        x = x + m * offset_norm(y, W(p + "norm1b"), eps)
        if layer["mlp"] is not None:
            x = x + m * offset_norm(mlp(offset_norm(x, W(p + "norm2"), eps), W, p + "mlp."), W(p + "norm2b"), eps)
        layers.append(x)
    logits = offset_norm(x, W("final.norm"), eps) @ W("embed").T * config["logit_scale"]
    return (logits, torch.stack(layers)) if want_layers else logits


# ---------------------------------------------------------------------------------------------- small random models
def make_config(width, vocab, layers, eps=1e-5, mult=0.8, logit_scale=0.5):
    return {"architecture": "Molitar", "layers": layers, "logit_scale": logit_scale, "norm": {"eps": eps},
            "residual_mult": mult, "vocab": vocab, "width": width}


def rotation(dims, base, scaling=None):
    return {"dims": dims, "base": base, **({"scaling": scaling} if scaling else {})}


def yarn(factor, original, fast=32.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def latent_layer(heads, dim, rot_dim, vdim, q_rank, kv_rank, base, scale, scaling=None, ff=None):
    return {"type": "latent_attention", "mlp": dense(ff), "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
        "rot": rotation(rot_dim, base, scaling)}}


def attention_layer(heads, kv_heads, dim, vdim, rot_dims, base, scale, softcap, v_mix, ff=None):
    return {"type": "attention", "mlp": dense(ff), "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap, "v_mix": v_mix,
        "rot": rotation(rot_dims, base)}}


def dense(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def tensor_shapes(config):
    """name -> shape of every tensor the design has for this configuration."""
    d = config["width"]
    s = {"embed": (config["vocab"], d), "final.norm": (d,)}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H = m["heads"]
        s.update({p + "norm1": (d,), p + "norm1b": (d,)})
        p += "mix."
        if layer["type"] == "latent_attention":
            s.update({p + "dq": (m["q_rank"], d), p + "dq.norm": (m["q_rank"],),
                      p + "uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                      p + "dkv": (m["kv_rank"] + m["rot_dim"], d), p + "dkv.norm": (m["kv_rank"],),
                      p + "uk": (H * m["dim"], m["kv_rank"]), p + "uv": (H * m["vdim"], m["kv_rank"]),
                      p + "o": (d, H * m["vdim"])})
        else:
            for n, rows in (("q", H * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                s.update({p + n: (rows, d), p + n + ".b": (rows,)})
            if m.get("v_mix"):
                s[p + "vmix"] = ()
            s.update({p + "sink": (H,), p + "g": (H * m["vdim"], d), p + "o": (d, H * m["vdim"])})
        if layer["mlp"] is not None:
            p, ff = f"l{i}.", layer["mlp"]["ff"]
            s.update({p + "norm2": (d,), p + "norm2b": (d,), p + "mlp.gate": (ff, d), p + "mlp.up": (ff, d), p + "mlp.down": (d, ff)})
    return s


def make_weights(config, seed):
    """Seeded random bf16 tensors: rows of unit gain, norm weights around zero (the latents' around one), biases spread over
    +-1, sinks around 1, mixing factors between 0.2 and 0.8."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in sorted(tensor_shapes(config).items()):
        t = torch.randn(shape, generator=g)
        if name.endswith("vmix"):
            t = 0.2 + 0.6 * torch.rand((), generator=g)
        elif len(shape) == 2:
            t = t * (1.0 if name == "embed" else shape[1] ** -0.5)
        elif name.endswith(("dq.norm", "dkv.norm")):
            t = 1.0 + 0.2 * t
        elif "norm" in name:
            t = 0.2 * t
        elif name.endswith("sink"):
            t = 1.0 + t
        out[name] = t.to(torch.bfloat16)
    return out
