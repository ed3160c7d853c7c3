"""The Molitar decoder for the hybrid runner: its config.json and tensor names.

Two token mixers in any order, each with norms before and after it and optionally followed by a gated feed-forward with
norms of its own: ``latent_attention`` (keys and values of all heads from one cached latent per token) and ``attention``
(grouped queries, biases, soft-capped scores, a sink per head, an output gate, values mixed with those of the first such
layer).  The embedding table is the output projection.
"""
import zlib

import torch

from . import hybrid
from .hybrid import HeadRows

_MLP_ACTS = {"dense": hybrid.ACT_SILU}


def _rotation(rot):
    """(frequencies, factor of cos and sin) of a mixer's ``rot`` entry."""
    if rot.get("scaling"):
        s = rot["scaling"]
        return hybrid.yarn_frequencies(rot["dims"], rot["base"], s["factor"], s["original"], s["fast"], s["slow"])
    return [float(rot["base"]) ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)], 1.0


def _heads(layer):
    """Row layouts of a mixer's heads: (query / key, value); of a latent mixer (unrotated, rotated, value)."""
    m = layer["mixer"]
    if layer["type"] == "latent_attention":
        return HeadRows(m["dim"]), HeadRows(m["rot_dim"], m["rot_dim"]), HeadRows(m["vdim"])
    return HeadRows(m["dim"], m["rot"]["dims"]), HeadRows(m["vdim"])


def _branch(layer):
    m = layer["mixer"]
    freq, amp = _rotation(m["rot"])
    if layer["type"] == "latent_attention":
        if m["rot"]["dims"] != m["rot_dim"]:
            raise ValueError("the rotation covers the rotated part of a head")
        plain, rot, value = _heads(layer)
        return hybrid.Branch(hybrid.LATENT, dim=plain.rows, vdim=value.rows, heads=m["heads"], rank=m["kv_rank"], q_rank=m["q_rank"],
                             rot_dims=rot.rot_rows, inv_freq=rot.pad_frequencies(freq), rot_scale=amp, score_scale=m["scale"])
    if layer["type"] == "attention":
        head, value = _heads(layer)
        flags = hybrid.SINK | hybrid.OUT_GATE | (hybrid.VALUE_MIX if m.get("v_mix") else 0)
        return hybrid.Branch(hybrid.ATTENTION, dim=head.rows, vdim=value.rows, heads=m["heads"], kv_heads=m["kv_heads"],
                             rot_dims=head.rot_rows, inv_freq=head.pad_frequencies(freq), rot_scale=amp, flags=flags,
                             score_scale=m["scale"], softcap=m.get("softcap") or 0.0)
    raise ValueError(f"unknown mixer type {layer['type']!r}")


def parse_config(config):
    """config.json (parsed) -> HybridConfig; head sizes are those of the runner's padded heads (hybrid.HeadRows)."""
    layers, mixed = [], set()
    for layer in config["layers"]:
        mlp = layer["mlp"]
        if mlp is not None and mlp["kind"] not in _MLP_ACTS:
            raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
        b = _branch(layer)
        if b.flags & hybrid.VALUE_MIX:
            mixed.add((b.kv_heads, layer["mixer"]["vdim"]))
        flags = hybrid.POST_NORM | (hybrid.IN_BIAS if b.kind == hybrid.ATTENTION else 0)
        layers.append(hybrid.Layer([b], mlp["ff"] if mlp else 0, _MLP_ACTS[mlp["kind"]] if mlp else 0, flags))
    if len(mixed) > 1:
        raise ValueError("layers that mix values have the same value heads")
    return hybrid.HybridConfig(config["width"], config["vocab"], config["norm"]["eps"], 1.0, layers, config["residual_mult"],
                               config["logit_scale"])


def _columns(w, heads):
    """Input columns of an output projection, moved and padded like the rows that feed them."""
    return heads.place(w.t()).t()


def _branch_weights(layer, t):
    """``t(name)``: tensor of the layer's mixer."""
    m = layer["mixer"]
    if layer["type"] == "latent_attention":
        plain, rot, value = _heads(layer)
        H, D, R = m["heads"], m["dim"], m["rot_dim"]
        uq = t("uq").view(H, D + R, -1)
        uq = torch.cat([rot.place(uq[:, D:].reshape(H * R, -1)).view(H, rot.rows, -1),
                        plain.place(uq[:, :D].reshape(H * D, -1)).view(H, plain.rows, -1)], 1)
        down = t("dkv")
        return {"inputs": [t("dq"), down[:m["kv_rank"]], rot.place(down[m["kv_rank"]:])], "out": _columns(t("o"), value),
                "q_norm": t("dq.norm"), "k_norm": t("dkv.norm"), "uq": uq.reshape(H * (rot.rows + plain.rows), -1),
                "uk": plain.place(t("uk")), "uv": value.place(t("uv"))}
    head, value = _heads(layer)
    return {"inputs": [head.place(t("q")), head.place(t("k")), value.place(t("v")), value.place(t("g"))],
            "biases": [head.place(t("q.b")), head.place(t("k.b")), value.place(t("v.b")), None],
            "out": _columns(t("o"), value), "sink": t("sink"), **({"value_mix": t("vmix")} if m.get("v_mix") else {})}


def _offset(w):
    """Norm weights are stored as differences from one."""
    return 1.0 + w.float()


def load_weights(runner, config, tensors):
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        ff = {}
        if layer["mlp"] is not None:
            ff = {"norm2": _offset(tensors[p + "norm2"]), "norm2_post": _offset(tensors[p + "norm2b"]),
                  **{n: tensors[f"{p}mlp.{n}"] for n in ("gate", "up", "down")}}
        runner.load_layer(i, _offset(tensors[p + "norm1"]), [_branch_weights(layer, lambda n: tensors[f"{p}mix.{n}"])],
                          norm1_post=_offset(tensors[p + "norm1b"]), **ff)
    embed = tensors["embed"]
    runner.load_head(embed, _offset(tensors["final.norm"]), embed)


def build(config, tensors, dtype=torch.bfloat16, **sizes):
    """A HybridRunner with this checkpoint's weights; ``sizes``: max_batch, max_len, ... of HybridRunner."""
    runner = hybrid.HybridRunner(parse_config(config), dtype=dtype, **sizes)
    load_weights(runner, config, tensors)
    return runner


def tensor_shapes(config):
    """name -> shape of every tensor of a checkpoint."""
    d = config["width"]
    out = {"embed": (config["vocab"], d), "final.norm": (d,)}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H = m["heads"]
        if layer["type"] == "latent_attention":
            mats = {"dq": (m["q_rank"], d), "uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]), "dkv": (m["kv_rank"] + m["rot_dim"], d),
                    "uk": (H * m["dim"], m["kv_rank"]), "uv": (H * m["vdim"], m["kv_rank"]), "dq.norm": (m["q_rank"],),
                    "dkv.norm": (m["kv_rank"],)}
        else:
            rows = {"q": H * m["dim"], "k": m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"]}
            mats = {**{n: (r, d) for n, r in rows.items()}, **{n + ".b": (r,) for n, r in rows.items()}, "g": (H * m["vdim"], d),
                    "sink": (H,), **({"vmix": ()} if m.get("v_mix") else {})}
        out.update({f"{p}mix.{n}": s for n, s in mats.items()})
        out.update({p + "mix.o": (d, H * m["vdim"]), p + "norm1": (d,), p + "norm1b": (d,)})
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            out.update({p + "norm2": (d,), p + "norm2b": (d,), f"{p}mlp.gate": (ff, d), f"{p}mlp.up": (ff, d), f"{p}mlp.down": (d, ff)})
    return out


class RandomTensors:
    """Seeded random bf16 checkpoint tensors, made on ``device`` when asked for: matrices of unit gain, norms around one."""

    def __init__(self, config, seed, device):
        self.shapes, self.seed, self.device = tensor_shapes(config), seed, device

    def __getitem__(self, name):
        shape = self.shapes[name]
        g = torch.Generator(device=self.device).manual_seed(self.seed * 1000003 + zlib.crc32(name.encode()))
        t = torch.randn(shape, generator=g, device=self.device)
        if len(shape) == 2:
            t *= shape[1] ** -0.5
        elif name.endswith(("dq.norm", "dkv.norm")):
            t = 1.0 + 0.1 * t
        elif "norm" in name:
            t = 0.1 * t
        elif name.endswith("vmix"):
            t = torch.full_like(t, 0.5)
        return t.to(torch.bfloat16)
