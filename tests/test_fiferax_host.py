"""Host side of the hybrid decoders and of the Fiferax design: configuration, weight fusion, step planning, registry (no GPU)."""
import random

import pytest
import torch

from oracle import fiferax as of


@pytest.fixture(scope="module", autouse=True)
def built():
    import __graft_entry__ as g
    g.build()


def small_config():
    return of.make_config(96, 133, [
        of.gru_layer(40, ff=100), of.delta_layer(3, 32),
        of.parallel_layer(6, 3, 32, 9, 16, 5000.0, 0.21, 3, 24, 40, [0.5, 0.9, 0.97], 0.7, 1.3, ff=72)], eps=1e-4, scale=1.7)


def test_configuration_carries_every_size_and_constant():
    from teenygrad_b200 import fiferax, hybrid
    c = fiferax.parse_config(small_config(), lambda i: 5)
    assert (c.width, c.vocab, c.eps, c.embed_scale) == (96, 133, 1e-4, 1.7)
    gru, delta, par = c.layers
    assert (gru.ff, gru.act, gru.branches[0].kind, gru.branches[0].dim) == (100, hybrid.ACT_GELU_TANH, hybrid.MIN_GRU, 40)
    assert (delta.ff, delta.branches[0].heads, delta.branches[0].dim, delta.branches[0].rank) == (0, 3, 32, 5)
    a, r = par.branches
    assert (a.heads, a.kv_heads, a.dim, a.window, a.rot_dims, a.rot_base, a.score_scale, a.out_scale) == (6, 3, 32, 9, 16, 5000.0, 0.21, 0.7)
    assert a.flags == hybrid.QK_NORM | hybrid.KEYS_ARE_VALUES
    assert (r.heads, r.dim, r.vdim, r.decay, r.out_scale) == (3, 24, 40, (0.5, 0.9, 0.97), 1.3)
    assert a.input_sizes() == [192, 96] and r.input_sizes() == [72, 72, 120, 120] and r.output_size() == 120


@pytest.mark.parametrize("spoil", ["mixer", "mlp", "decay"])
def test_unknown_parts_are_refused(spoil):
    from teenygrad_b200 import fiferax
    cfg = small_config()
    if spoil == "mixer":
        cfg["layers"][1]["type"] = "something"
    elif spoil == "mlp":
        cfg["layers"][0]["mlp"]["kind"] = "other"
    else:
        cfg["layers"][2]["mixer"]["right"]["decay"].pop()
    with pytest.raises(ValueError):
        fiferax.parse_config(cfg, lambda i: 5)


def test_tensor_names_and_shapes_are_the_designs():
    from teenygrad_b200 import fiferax
    assert fiferax.tensor_shapes(small_config(), 5) == of.tensor_shapes(small_config(), 5)


def test_fused_weights_keep_every_part_at_a_multiple_of_eight():
    from teenygrad_b200 import hybrid
    g = torch.Generator().manual_seed(0)
    a, b = torch.randn(5, 11, generator=g), torch.randn(9, 11, generator=g)
    f = hybrid.fuse_rows([a, b], torch.float32)
    assert f.shape == (24, 16) and torch.equal(f[:5, :11], a) and torch.equal(f[8:17, :11], b)
    assert float(f.abs().sum()) == pytest.approx(float(a.abs().sum() + b.abs().sum()), rel=1e-6)
    c = hybrid.fuse_columns([a.t(), b.t()], torch.float32)
    assert c.shape == (11, 24) and torch.equal(c[:, :5], a.t()) and torch.equal(c[:, 8:17], b.t())
    gate, up = torch.randn(70, 12, generator=g), torch.randn(70, 12, generator=g)
    w = hybrid.interleave_glu(gate, up, torch.float32).view(2, 2, 64, 16)
    assert torch.equal(w[0, 0, :, :12], gate[:64]) and torch.equal(w[1, 1, :6, :12], up[64:])
    assert not w[1, :, 6:].any() and not w[..., 12:].any()


def test_step_planning_covers_every_token_and_row_once():
    from teenygrad_b200.hybrid import plan_steps
    rng = random.Random(3)
    for _ in range(200):
        entries = []
        for _ in range(rng.randint(1, 5)):
            n = rng.randint(1, 40)
            entries.append((n, sorted(rng.sample(range(n), rng.randint(0, n)))))
        max_tokens, max_rows = rng.randint(1, 30), rng.randint(1, 12)
        at, rows = [0] * len(entries), [[] for _ in entries]
        for step in plan_steps(entries, max_tokens, max_rows):
            assert step and sum(c for _, _, c, _ in step) <= max_tokens and sum(len(w) for *_, w in step) <= max_rows
            assert len({e for e, *_ in step}) == len(step)
            for e, first, count, want in step:
                assert first == at[e] and count > 0 and all(first <= p < first + count for p in want)
                at[e] += count
                rows[e] += want
        assert at == [n for n, _ in entries] and rows == [w for _, w in entries]


def test_registry_picks_the_model_by_its_architecture():
    from teenygrad_b200 import models
    assert models.architecture({"architecture": "Fiferax"}) == "Fiferax"
    assert models.architecture({"architectures": ["Qwen3ForCausalLM"]}) == "Qwen3ForCausalLM"
    with pytest.raises(ValueError, match="no model"):
        models.architecture({"architecture": "Nothing"})


def test_unsupported_sizes_and_dtypes_are_refused():
    from teenygrad_b200 import fiferax, hybrid
    cfg = fiferax.parse_config(small_config(), lambda i: 5)
    with pytest.raises(ValueError, match="bfloat16 or float32"):
        hybrid.HybridRunner(cfg, max_batch=1, max_len=8, dtype=torch.float16)
    cfg.layers[1].branches[0].dim = cfg.layers[1].branches[0].vdim = 400  # larger than any state kernel takes
    with pytest.raises(ValueError, match="unsupported"):
        hybrid.HybridRunner(cfg, max_batch=1, max_len=8)


def test_command_line_arguments():
    from teenygrad_b200.generate import parse_args
    a = parse_args(["--model", "m", "--prompt", "1,2,3", "--prompt", "7", "--dtype", "float32", "--temperature", "0.5"])
    assert a.prompt == [[1, 2, 3], [7]] and a.dtype == "float32" and a.temperature == 0.5


def test_oracle_attention_forms_agree():
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(30, h, 8, generator=g, dtype=torch.float64) for h in (4, 2, 2))
    for w in (1, 7, 29, 100):
        assert torch.allclose(of.window_attention(q, k, v, 0.4, w), of.window_attention_fast(q, k, v, 0.4, w), atol=1e-12)


def test_oracle_gru_candidate_is_continuous_at_zero_and_positive():
    u = torch.tensor([[-1e-9], [0.0], [1e-9], [-40.0], [3.0]], dtype=torch.float64)
    out = torch.cat([of.min_gru(torch.full((1, 1), 60.0, dtype=torch.float64), x[None])[0] for x in u])
    assert torch.allclose(out[:3], torch.full((3, 1), 0.5, dtype=torch.float64), atol=1e-8) and out[3] > 0 and out[4] == 3.5
