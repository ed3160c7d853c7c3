"""Host side of the Molitar design and of full / latent attention in the hybrid runner: configuration, head layouts, weight
preparation, registry, and the float64 restatement's own consistency (no GPU)."""
import math

import pytest
import torch

from oracle import molitar as om

F64 = torch.float64


@pytest.fixture(scope="module", autouse=True)
def built():
    import __graft_entry__ as g
    g.build()


def rnd(seed, *shape):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64)


def small_config():
    return om.make_config(72, 111, [
        om.attention_layer(6, 2, 22, 12, 10, 700.0, 0.3, 6.0, True, ff=50),
        om.latent_layer(3, 20, 12, 28, 18, 34, 900.0, 0.2, om.yarn(8.0, 64, 20.0, 2.0)),
        om.attention_layer(4, 4, 16, 12, 16, 50.0, 0.4, 30.0, False)], eps=1e-3, mult=1.3, logit_scale=2.0)


def test_configuration_carries_every_size_and_constant():
    from teenygrad_b200 import hybrid, molitar
    c = molitar.parse_config(small_config())
    assert (c.width, c.vocab, c.eps, c.residual_mult, c.logit_scale, c.embed_scale) == (72, 111, 1e-3, 1.3, 2.0, 1.0)
    a, lat, b = (layer.branches[0] for layer in c.layers)
    assert [layer.ff for layer in c.layers] == [50, 0, 0] and c.layers[0].act == hybrid.ACT_SILU
    assert [layer.flags for layer in c.layers] == [hybrid.POST_NORM | hybrid.IN_BIAS, hybrid.POST_NORM, hybrid.POST_NORM | hybrid.IN_BIAS]
    assert (a.kind, a.heads, a.kv_heads, a.window, a.score_scale, a.softcap) == (hybrid.ATTENTION, 6, 2, 0, 0.3, 6.0)
    assert a.flags == hybrid.SINK | hybrid.OUT_GATE | hybrid.VALUE_MIX and b.flags == hybrid.SINK | hybrid.OUT_GATE
    assert (a.rot_dims, a.dim, a.vdim) == (16, 32, 16) and (b.rot_dims, b.dim) == (16, 16)
    assert a.inv_freq[:5] == [700.0 ** (-2 * i / 10) for i in range(5)] and a.inv_freq[5:] == [0.0] * 3
    assert (lat.kind, lat.heads, lat.rank, lat.q_rank, lat.rot_dims, lat.dim, lat.vdim) == (hybrid.LATENT, 3, 34, 18, 16, 24, 32)
    assert lat.rot_scale == 0.1 * math.log(8.0) + 1.0 and lat.input_sizes() == [18, 34, 16] and lat.output_size() == 96
    assert a.input_sizes() == [192, 64, 32, 96]


@pytest.mark.parametrize("spoil", ["mixer", "mlp", "rotation", "values"])
def test_unknown_parts_are_refused(spoil):
    from teenygrad_b200 import molitar
    cfg = small_config()
    if spoil == "mixer":
        cfg["layers"][1]["type"] = "something"
    elif spoil == "mlp":
        cfg["layers"][0]["mlp"]["kind"] = "other"
    elif spoil == "rotation":
        cfg["layers"][1]["mixer"]["rot"]["dims"] = 8
    else:
        cfg["layers"][2]["mixer"]["v_mix"] = True  # other value heads than the first such layer
    with pytest.raises(ValueError):
        molitar.parse_config(cfg)


def test_tensor_names_and_shapes_are_the_designs():
    from teenygrad_b200 import molitar
    assert molitar.tensor_shapes(small_config()) == om.tensor_shapes(small_config())


def test_registry_knows_the_design():
    from teenygrad_b200 import models
    assert models.architecture({"architecture": "Molitar"}) == "Molitar"


def test_unsupported_sizes_are_refused():
    from teenygrad_b200 import hybrid, molitar
    for key, value in (("rank", 1100), ("dim", 300), ("dim", 12)):
        cfg = molitar.parse_config(small_config())
        setattr(cfg.layers[1].branches[0], key, value)
        with pytest.raises(ValueError, match="unsupported"):
            hybrid.HybridRunner(cfg, max_batch=1, max_len=8)


@pytest.mark.parametrize("dims,base,scaling", [(16, 1e4, (4.0, 512, 32.0, 1.0)), (64, 5e5, (1.0, 4096, 32.0, 1.0)), (12, 30.0, (16.0, 64, 8.0, 3.0)),
                                               (8, 10.0, (2.5, 7, 1.0, 0.9)), (32, 1e6, (40.0, 1 << 20, 2.0, 1.5))])
def test_stretched_frequencies(dims, base, scaling):
    from teenygrad_b200 import hybrid
    f, amp = hybrid.yarn_frequencies(dims, base, *scaling)
    want, want_amp = om.rotation_frequencies(dims, base, om.yarn(*scaling))
    assert f == pytest.approx(want, rel=1e-12) and amp == pytest.approx(want_amp)
    plain, one = om.rotation_frequencies(dims, base)
    assert one == 1.0 and all(w <= p * (1 + 1e-12) and w >= p / scaling[0] * (1 - 1e-12) for w, p in zip(want, plain))


def rotate_half(x, pos, freq, amp):
    """The kernels' rotation: i with i + half."""
    h = len(freq)
    a = pos.to(F64)[:, None] * torch.tensor(freq, dtype=F64)
    c, s = amp * torch.cos(a)[:, None], amp * torch.sin(a)[:, None]
    u, v = x[..., :h], x[..., h:2 * h]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * h:]], -1)


@pytest.mark.parametrize("dim,rot", [(24, 24), (22, 10), (64, 32), (9, 2), (16, 0)])
def test_head_rows_keep_the_scores(dim, rot):
    """Neighbour pairs rotated in the checkpoint's order = halves rotated in the runner's order."""
    from teenygrad_b200 import hybrid
    rows = hybrid.HeadRows(dim, rot)
    assert rows.rows % 8 == 0 and rows.rows >= dim
    wq, wk, x = rnd(1, 3 * dim, 10), rnd(2, 3 * dim, 10), rnd(3, 7, 10)
    pos = torch.tensor([0, 1, 5, 100, 101, 4000, 4001])
    scaling = om.yarn(3.0, 100) if rot else None
    freq, amp = om.rotation_frequencies(rot, 50.0, scaling) if rot else ([], 1.0)

    def scores(q, k):
        return torch.einsum("ihd,jhd->hij", q, k)

    turn = lambda w: om.rotary_pairs((x @ w.T).view(7, 3, dim), pos, rot, 50.0, scaling) if rot else (x @ w.T).view(7, 3, dim)  # noqa: E731
    half = lambda w: rotate_half((x @ rows.place(w).T).view(7, 3, rows.rows), pos, rows.pad_frequencies(freq), amp)  # noqa: E731
    assert torch.allclose(scores(turn(wq), turn(wk)), scores(half(wq), half(wk)), atol=1e-9)
    assert torch.equal(rows.place(wq[:, 0]), rows.place(wq)[:, 0])


def test_latent_weights_expand_and_absorb_alike():
    """EXPAND makes every head's key [rotated, plain] and value from a cache row; ABSORB and VALUE_UP give the same scores and
    outputs in the latent space."""
    from teenygrad_b200 import hybrid
    b = hybrid.Branch(hybrid.LATENT, dim=16, vdim=8, heads=3, rank=21, q_rank=9, rot_dims=16)
    uk, uv = rnd(1, 3 * 16, 21), rnd(2, 3 * 8, 21)
    expand, absorb, up = hybrid.latent_weights(b, uk, uv, F64)
    c, shared, q = rnd(3, 5, 21), rnd(4, 5, 16), rnd(5, 4, 3, 32)
    row = torch.cat([c, torch.zeros(5, 3, dtype=F64), shared], 1)
    made = row @ expand.T
    k, v = made[:, :3 * 32].view(5, 3, 32), made[:, 3 * 32:].view(5, 3, 8)
    assert torch.equal(k[..., :16], shared[:, None].expand(5, 3, 16))
    assert torch.allclose(k[..., 16:], (c @ uk.T).view(5, 3, 16)) and torch.allclose(v, (c @ uv.T).view(5, 3, 8))
    qa = torch.cat([torch.einsum("thk,hnk->thn", q[..., 16:], absorb), q[..., :16]], -1)
    s = torch.einsum("ihd,jhd->hij", q, k)
    assert torch.allclose(torch.einsum("ihd,jd->hij", qa, row), s)
    p = torch.softmax(s, -1)
    out = torch.einsum("thk,hnk->thn", torch.einsum("hij,jd->ihd", p, row[:, :24]), up)
    assert torch.allclose(out, torch.einsum("hij,jhd->ihd", p, v))


# ------------------------------------------------------------------------------------- the restatement itself
def test_oracle_attention_forms_agree():
    q, k, v = rnd(1, 25, 4, 8), rnd(2, 25, 2, 8), rnd(3, 25, 2, 5)
    sink = rnd(4, 4)
    for cap, s in ((None, None), (2.0, None), (None, sink), (0.7, 3 * sink)):
        assert torch.allclose(om.causal_attention(q, k, v, 0.4, cap, s), om.causal_attention_fast(q, k, v, 0.4, cap, s), atol=1e-12)


def test_oracle_sink_takes_weight_and_nothing_else():
    q, k, v = rnd(1, 6, 1, 4), rnd(2, 6, 1, 4), torch.ones(6, 1, 3, dtype=F64)
    out = om.causal_attention(q, k, v, 0.5, None, torch.tensor([1.5], dtype=F64))
    for i in range(6):
        e = torch.exp((k[:i + 1, 0] @ q[i, 0]) * 0.5).sum()
        assert torch.allclose(out[i, 0], (e / (e + math.exp(1.5))).expand(3))
    assert torch.allclose(om.causal_attention(q, k, v, 0.5, None, torch.tensor([-800.0], dtype=F64)), v[:, :, :].expand(6, 1, 3))


def test_oracle_mixers_match_their_attention_loops():
    cfg = small_config()
    w = om.make_weights(cfg, 3)
    h = rnd(5, 9, 72)
    W = lambda n: w[n].to(F64)  # noqa: E731
    for i, layer in enumerate(cfg["layers"]):
        for shared in ({}, {"v": rnd(6, 9, 2, 12)} if layer["type"] == "attention" else {}):
            mix = om.MIXERS[layer["type"]]
            a, b = (mix(h, W, f"l{i}.mix.", layer["mixer"], 1e-3, dict(shared), fast) for fast in (True, False))
            assert torch.allclose(a, b, atol=1e-11)


def test_oracle_rotation_is_a_rotation_scaled():
    x = rnd(1, 4, 2, 12)
    pos = torch.tensor([0, 3, 50, 900])
    y = om.rotary_pairs(x, pos, 8, 100.0, om.yarn(4.0, 32))
    amp = 0.1 * math.log(4.0) + 1.0
    assert torch.equal(y[..., 8:], x[..., 8:]) and torch.allclose(y[0, :, :8], amp * x[0, :, :8])
    assert torch.allclose(y[..., :8].pow(2).sum(-1), amp ** 2 * x[..., :8].pow(2).sum(-1))


def test_every_mechanism_shows_in_the_logits():
    """The random models the GPU tests use are sensitive to each part (a mistake planted here, in the restatement)."""
    import copy
    import test_gpu_molitar as gpu
    cfg, w, toks, want = gpu.case("a")
    t = toks[90]

    def change(config=None, weights=None):
        c, v = copy.deepcopy(cfg), dict(w)
        if config:
            for layer in c["layers"]:
                config(layer)
        if weights:
            for n in v:
                v[n] = weights(n, v[n])
        return float((om.forward(c, v, t) - want[90]).pow(2).mean().sqrt() / want[90].pow(2).mean().sqrt())

    def no_cap(layer):
        if layer["type"] == "attention":
            layer["mixer"]["softcap"] = 1e6

    def no_yarn(layer):
        layer["mixer"]["rot"].pop("scaling", None)

    def no_mix(layer):
        if layer["type"] == "attention":
            layer["mixer"]["v_mix"] = False

    ending = lambda e, f: lambda n, x: f(x) if n.endswith(e) else x  # noqa: E731
    for what in (dict(config=no_cap), dict(config=no_yarn), dict(config=no_mix), dict(weights=ending("sink", lambda x: x - 50)),
                 dict(weights=ending(".g", lambda x: x * 0)), dict(weights=ending("k.b", lambda x: x * 0)),
                 dict(weights=ending("norm1b", lambda x: x * 0)), dict(weights=ending("dkv.norm", lambda x: x * 0 + 1))):
        assert change(**what) > 0.03, what
