"""Model registry: a checkpoint folder (config.json, model.safetensors) -> a runner, chosen by the configuration's
``architecture`` (or Hugging Face ``architectures``) entry."""
import json
import os

import torch

from .safetensors import SafeTensors


def _qwen3(config, tensors, dtype, **sizes):
    from . import qwen3
    if dtype != torch.bfloat16:
        raise ValueError("Qwen3 runs in bfloat16")
    rope = config.get("rope_theta") or config["rope_parameters"]["rope_theta"]
    cfg = qwen3.Qwen3Config(config["num_hidden_layers"], config["hidden_size"], config["num_attention_heads"],
                            config["num_key_value_heads"], config["head_dim"], config["intermediate_size"], config["vocab_size"],
                            config["rms_norm_eps"], rope, config.get("tie_word_embeddings", False))
    runner = qwen3.Qwen3Runner(cfg, **sizes)
    runner.load_state_dict(tensors)
    return runner


def _fiferax(config, tensors, dtype, **sizes):
    from . import fiferax
    return fiferax.build(config, tensors, dtype, **sizes)


def _molitar(config, tensors, dtype, **sizes):
    from . import molitar
    return molitar.build(config, tensors, dtype, **sizes)


REGISTRY = {"Qwen3ForCausalLM": _qwen3, "Fiferax": _fiferax, "Molitar": _molitar}


def architecture(config):
    names = [config["architecture"]] if "architecture" in config else config.get("architectures", [])
    for n in names:
        if n in REGISTRY:
            return n
    raise ValueError(f"no model for architecture {names}; known: {sorted(REGISTRY)}")


def load(path, dtype=torch.bfloat16, **sizes):
    """``sizes``: the runner's capacities (max_batch, max_len, max_tokens, max_new_tokens, ...)."""
    with open(os.path.join(path, "config.json")) as f:
        config = json.load(f)
    return REGISTRY[architecture(config)](config, SafeTensors(path), dtype, **sizes)
