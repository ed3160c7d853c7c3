"""The Fiferax decoder for the hybrid runner: its config.json and tensor names.

Three token mixers in any order, each behind a pre-norm and optionally followed by a gated feed-forward:
``general_delta`` (generalized delta rule), ``parallel`` (sliding-window attention whose values are the raw keys, beside
scalar-decay linear attention) and ``mingru``.
"""
import math
import zlib

import torch

from . import hybrid

DECAY_COEF = math.exp(-0.5)  # w = exp(-exp(-1/2) sigmoid(...))
UNIT_EPS = 1e-6              # u = k / sqrt(sum k^2 + 1e-6)

_MLP_ACTS = {"dense": hybrid.ACT_GELU_TANH}


def _branches(layer, rank):
    m = layer["mixer"]
    kind = layer["type"]
    if kind == "general_delta":
        return [hybrid.Branch(hybrid.DELTA, dim=m["dim"], vdim=m["dim"], heads=m["heads"], rank=rank, decay_coef=DECAY_COEF,
                              unit_eps=UNIT_EPS)]
    if kind == "mingru":
        return [hybrid.Branch(hybrid.MIN_GRU, dim=m["width"])]
    if kind == "parallel":
        a, r = m["left"], m["right"]
        if a["vdim"] != a["dim"]:
            raise ValueError("values that are the keys have the keys' size")
        if len(r["decay"]) != r["heads"]:
            raise ValueError("one decay per head")
        return [hybrid.Branch(hybrid.ATTENTION, dim=a["dim"], vdim=a["vdim"], heads=a["heads"], kv_heads=a["kv_heads"],
                              window=a["mask"]["size"], rot_dims=a["rot"]["dims"], rot_base=a["rot"]["base"],
                              flags=hybrid.QK_NORM | hybrid.KEYS_ARE_VALUES, score_scale=a["scale"], out_scale=m["left_scale"]),
                hybrid.Branch(hybrid.DECAY, dim=r["dim"], vdim=r["vdim"], heads=r["heads"], decay=tuple(r["decay"]),
                              out_scale=m["right_scale"])]
    raise ValueError(f"unknown mixer type {kind!r}")


def parse_config(config, rank_of):
    """config.json (parsed) -> HybridConfig.  ``rank_of(layer)``: rows of that layer's decay factor ``w1``, a size that only
    its tensor's shape gives."""
    layers = []
    for i, layer in enumerate(config["layers"]):
        mlp = layer["mlp"]
        if mlp is not None and mlp["kind"] not in _MLP_ACTS:
            raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
        rank = rank_of(i) if layer["type"] == "general_delta" else 0
        layers.append(hybrid.Layer(_branches(layer, rank), mlp["ff"] if mlp else 0, _MLP_ACTS[mlp["kind"]] if mlp else 0))
    return hybrid.HybridConfig(config["width"], config["vocab"], config["norm"]["eps"], config["embedding"]["scale"], layers)


def _branch_weights(kind, t):
    """``t(name)``: tensor of the layer's mixer."""
    if kind == "general_delta":
        return [{"inputs": [t(n) for n in ("r", "k", "v", "a", "g", "w1")], "out": t("o"), "low": t("w2"), "decay_bias": t("w0"),
                 "rate_bias": t("a.b"), "o_norm": t("norm")}]
    if kind == "mingru":
        return [{"inputs": [t(n) for n in "zxg"], "out": t("o"), "z_bias": t("z.b"), "x_bias": t("x.b")}]
    return [{"inputs": [t("left.q"), t("left.k")], "out": t("left.o"), "q_norm": t("left.q.norm"), "k_norm": t("left.k.norm")},
            {"inputs": [t("right." + n) for n in "qkvg"], "out": t("right.o"), "o_norm": t("right.norm")}]


def load_weights(runner, config, tensors):
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        ff = {}
        if layer["mlp"] is not None:
            ff = {"norm2": tensors[p + "norm2"], **{n: tensors[f"{p}mlp.{n}"] for n in ("gate", "up", "down")}}
        runner.load_layer(i, tensors[p + "norm1"], _branch_weights(layer["type"], lambda n: tensors[f"{p}mix.{n}"]), **ff)
    runner.load_head(tensors["embed"], tensors["final.norm"], tensors["head"])


def build(config, tensors, dtype=torch.bfloat16, **sizes):
    """A HybridRunner with this checkpoint's weights; ``sizes``: max_batch, max_len, ... of HybridRunner."""
    cfg = parse_config(config, lambda i: tensors[f"l{i}.mix.w1"].shape[0])
    runner = hybrid.HybridRunner(cfg, dtype=dtype, **sizes)
    load_weights(runner, config, tensors)
    return runner


def tensor_shapes(config, rank):
    """name -> shape of every tensor of a checkpoint; ``rank``: rows of the decay factors ``w1``."""
    d = config["width"]
    out = {"embed": (config["vocab"], d), "final.norm": (d,), "head": (config["vocab"], d)}
    for i, layer in enumerate(config["layers"]):
        out[f"l{i}.norm1"] = (d,)
        for b, side in zip(_branches(layer, rank), ("left.", "right.") if layer["type"] == "parallel" else ("",)):
            p = f"l{i}.mix.{side}"
            names = {hybrid.ATTENTION: "qk", hybrid.DELTA: "rkvag", hybrid.DECAY: "qkvg", hybrid.MIN_GRU: "zxg"}[b.kind]
            out.update({p + n: (rows, d) for n, rows in zip(names, b.input_sizes())})
            out[p + "o"] = (d, b.output_size())
            n = b.heads * b.dim
            if b.kind == hybrid.ATTENTION:
                out.update({p + "q.norm": (b.dim,), p + "k.norm": (b.dim,)})
            elif b.kind == hybrid.MIN_GRU:
                out.update({p + "z.b": (n,), p + "x.b": (n,)})
            else:
                out[p + "norm"] = (b.output_size(),)
            if b.kind == hybrid.DELTA:
                out.update({p + "w1": (rank, d), p + "w2": (n, rank), p + "w0": (n,), p + "a.b": (n,)})
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            out.update({f"l{i}.norm2": (d,), f"l{i}.mlp.gate": (ff, d), f"l{i}.mlp.up": (ff, d), f"l{i}.mlp.down": (d, ff)})
    return out


class RandomTensors:
    """Seeded random bf16 checkpoint tensors, made on ``device`` when asked for: matrices of unit gain, norms around 1."""

    def __init__(self, config, seed, device, rank):
        self.shapes, self.seed, self.device = tensor_shapes(config, rank), seed, device

    def __getitem__(self, name):
        shape = self.shapes[name]
        g = torch.Generator(device=self.device).manual_seed(self.seed * 1000003 + zlib.crc32(name.encode()))
        t = torch.randn(*shape, generator=g, device=self.device)
        if len(shape) == 2:
            t *= shape[1] ** -0.5
        elif "norm" in name:
            t = 1.0 + 0.1 * t
        return t.to(torch.bfloat16)
