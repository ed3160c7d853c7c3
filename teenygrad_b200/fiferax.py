"""The Fiferax decoder for the hybrid runner: its config.json and tensor names.

Three token mixers in any order, each behind a pre-norm and optionally followed by a gated feed-forward:
``general_delta`` (generalized delta rule), ``parallel`` (sliding-window attention whose values are the raw keys, beside
scalar-decay linear attention) and ``mingru``.
"""
import math

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
