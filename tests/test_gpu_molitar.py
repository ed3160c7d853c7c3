"""The Molitar decoder, full attention and latent attention on a GPU, against the plain float64 restatement in
oracle/molitar.py: every mechanism alone (through its own entry point), whole prompts, portions, token-by-token decoding,
unequal batches, reused slots, and generation through the runner, the command line and the trace replay."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import molitar as om

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF, F32, F64 = torch.bfloat16, torch.float32, torch.float64
DTYPES = pytest.mark.parametrize("dtype", [F32, BF], ids=["f32", "bf16"])


@pytest.fixture(scope="module", autouse=True)
def cuda():
    if not torch.cuda.is_available():
        pytest.skip("no CUDA device")
    yield
    from teenygrad_b200 import ops
    assert ops.device_error() == 0


def rnd(seed, *shape):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


def rel(got, want):
    return float((got.double().cpu() - want).abs().max() / want.abs().max())


def entries_of(lens, slots, pos=None):
    """Step table: the entries' rows follow one another."""
    row, out = 0, []
    for i, n in enumerate(lens):
        out.append((slots[i], pos[i] if pos else 0, row, n))
        row += n
    return out


def rotate_half(x, pos, freq, amp):
    h = len(freq)
    a = pos.to(F64)[:, None] * torch.tensor(freq, dtype=F64)
    c, s = amp * torch.cos(a)[:, None], amp * torch.sin(a)[:, None]
    u, v = x[..., :h], x[..., h:2 * h]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * h:]], -1)


# ------------------------------------------------------------------------------------------------ mechanisms alone
@DTYPES
@pytest.mark.parametrize("n", [96, 4096, 50])
def test_norm_behind_a_sublayer(dtype, n):
    from teenygrad_b200 import ops
    x, d, w, post = 5 * rnd(1, 33, n), 0.3 * rnd(2, 33, n).to(dtype), rnd(3, n), 1 + rnd(4, n)
    xd = x.cuda()
    y = ops.residual_rms_norm(xd, d.cuda(), w.cuda(), 1e-2, post.cuda(), 0.7)
    s = x.double() + 0.7 * om.rms(d.double(), 1e-2) * post.double()
    assert rel(xd, s) < 1e-6 and rel(y, om.rms(s, 1e-2) * w.double()) < (1e-5 if dtype == F32 else 5e-3)


@DTYPES
@pytest.mark.parametrize("heads,kv,dim,vdim,rot", [(4, 2, 64, 64, 32), (3, 1, 128, 40, 128), (2, 2, 20, 12, 6), (6, 3, 88, 56, 40), (2, 1, 80, 16, 0)])
@pytest.mark.parametrize("mode", ["plain", "keep", "mix"])
def test_positions_value_mixing_and_cache(dtype, heads, kv, dim, vdim, rot, mode):
    from teenygrad_b200 import ops
    lens, pos, slots = [9, 1, 4], [0, 30, 1900], [2, 0, 1]
    rows, cap = sum(lens), 1910
    q, k, v = (3 * rnd(i, rows, h, d) for i, (h, d) in enumerate(((heads, dim), (kv, dim), (kv, vdim))))
    q, k, v = q.to(dtype).cuda(), k.to(dtype).cuda(), v.to(dtype).cuda()
    freq, amp = om.rotation_frequencies(rot, 700.0, om.yarn(4.0, 200)) if rot else ([], 1.3)
    kc, vc = (torch.full((3, kv, cap, d), 7.0, dtype=dtype, device="cuda") for d in (dim, vdim))
    lam = torch.tensor([0.3]).to(BF).float()
    first = None if mode == "plain" else rnd(9, rows, kv * vdim).to(dtype).cuda()
    before = None if first is None else first.double().cpu()
    qin, kin, vin = q.double().cpu(), k.double().cpu(), v.double().cpu()
    table = entries_of(lens, slots, pos)
    ops.rope_cache(q, k, v, kc, vc, torch.tensor(freq).float().cuda() if rot else None, rot, ops.seq_table(table), max(lens), rot_scale=amp,
                   v_first=first, mix=lam.cuda() if mode == "mix" else None)
    p = torch.cat([torch.arange(n) + s for n, s in zip(lens, pos)])
    tol = 2e-4 if dtype == F32 else 5e-3
    turn = lambda x: rotate_half(x, p, freq, amp) if rot else x  # noqa: E731
    assert rel(q, turn(qin)) < tol
    if mode == "mix":
        vin = om.mix_values(vin, before.view(rows, kv, vdim), float(lam))
    if mode == "keep":
        assert torch.equal(first.double().cpu(), vin.reshape(rows, -1))
    wk = turn(kin)
    for slot, at, r0, n in table:
        assert rel(kc[slot, :, at:at + n].transpose(0, 1), wk[r0:r0 + n]) < tol
        assert rel(vc[slot, :, at:at + n].transpose(0, 1), vin[r0:r0 + n]) < tol
        kc[slot, :, at:at + n] = vc[slot, :, at:at + n] = 7.0
    assert bool((kc == 7.0).all()) and bool((vc == 7.0).all())  # nothing else was written


def planted(seed, T, heads, kv, dim, vdim):
    """Random queries and keys in which some queries match one key so well that it takes all the weight if it is visible: the
    first keys, far ones, those around tile borders, its own and the next one (which it must not see)."""
    q, k, v = rnd(seed, T, heads, dim), rnd(seed + 1, T, kv, dim), rnd(seed + 2, T, kv, vdim)
    for n, i in enumerate(range(3, T, 5)):
        j = (0, i + 1, i, 1, i - 64, i // 2, 63, 64, 127, 128, i - 1)[n % 11]
        if 0 <= j < T:
            q[i] = 4.0 * k[j].repeat_interleave(heads // kv, 0)
    return q, k, v


SHAPES = [(4, 1, 128, 128), (4, 2, 88, 56), (6, 2, 64, 64), (2, 2, 72, 120), (8, 1, 32, 48), (2, 1, 136, 24), (3, 3, 20, 12), (8, 2, 48, 128),
          (4, 4, 192, 128), (2, 1, 144, 64)]


@DTYPES
@pytest.mark.parametrize("heads,kv,dim,vdim", SHAPES)
@pytest.mark.parametrize("cuts", ["whole", "portions", "long", "decode"])
def test_full_attention(dtype, heads, kv, dim, vdim, cuts):
    """Soft cap (scores well into its bend), sinks (one that takes almost everything), gate; over the cache."""
    from teenygrad_b200 import ops
    T, cap, scale = 300, 3.0, 0.25
    q, k, v = (t.to(dtype) for t in planted(3, T, heads, kv, dim, vdim))
    gate = (2 * rnd(8, T, heads * vdim)).to(dtype)
    sink = torch.linspace(-2.0, 4.0, heads)
    want = om.causal_attention_fast(q.double(), k.double(), v.double(), scale, cap, sink.double())
    want = want * om.sigmoid(gate.double()).view(T, heads, vdim)
    kc, vc = (torch.full((3, kv, T + 5, d), float("nan"), dtype=dtype, device="cuda") for d in (dim, vdim))
    sizes = {"whole": [T], "portions": [2, 63, 64, 1, 65, 3, 2, 100], "long": [7, 129, 164], "decode": [T - 70] + [1] * 70}[cuts]
    at, out = 0, []
    for n in sizes:
        s = slice(at, at + n)
        kc[1, :, s], vc[1, :, s] = k[s].transpose(0, 1).cuda(), v[s].transpose(0, 1).cuda()
        out.append(ops.cached_attention(q[s].cuda(), kc, vc, scale, [(1, at, 0, n)], softcap=cap, sink=sink.cuda(), gate=gate[s].cuda()))
        at += n
    assert rel(torch.cat(out), want) < (2e-5 if dtype == F32 else 1.5e-2)


@pytest.mark.parametrize("cap,sinks,gated", [(0.0, False, False), (50.0, False, True), (0.0, True, False), (4.0, True, True)])
@pytest.mark.parametrize("D,V", [(128, 128), (192, 128), (96, 56)])
def test_full_attention_in_batches(cap, sinks, gated, D, V):
    """Unequal entries in one step: equal long ones in neighbouring slots, long ones with a past, short ones and single tokens."""
    from teenygrad_b200 import ops
    H, G, C = 4, 2, 700
    sink = torch.tensor([-1.0, 0.5, 2.0, 5.0]) if sinks else None
    full = {b: planted(20 * b + 1, C, H, G, D, V) for b in range(7)}
    full = {b: tuple(t.to(BF) for t in p) for b, p in full.items()}
    gate = {b: rnd(100 + b, C, H * V).to(BF) for b in range(7)}
    want = {b: om.causal_attention_fast(*(t.double() for t in p), 0.1, cap or None, sink.double() if sinks else None) for b, p in full.items()}
    kc, vc = (torch.stack([p[i].transpose(0, 1) for p in full.values()]).contiguous().cuda() for i in (1, 2))
    table = entries_of([260, 260, 260, 5, 1, 130, 40], [1, 2, 3, 0, 4, 6, 5], [0, 0, 0, 50, 699, 401, 30])
    q = torch.cat([full[s][0][p:p + n] for s, p, _, n in table])
    g = torch.cat([gate[s][p:p + n] for s, p, _, n in table]) if gated else None
    got = ops.cached_attention(q.cuda(), kc, vc, 0.1, table, softcap=cap, sink=sink.cuda() if sinks else None, gate=g.cuda() if gated else None)
    for s, p, r0, n in table:
        e = want[s][p:p + n]
        if gated:
            e = e * om.sigmoid(gate[s][p:p + n].double()).view(n, H, V)
        assert rel(got[r0:r0 + n], e) < 1.5e-2, (s, p)


@pytest.mark.parametrize("D,V", [(128, 128), (192, 64)])
@pytest.mark.parametrize("cap", [0.0, 2.0, 400.0])
def test_full_attention_many_work_items(D, V, cap):
    """More (query tile, head, sequence) items than the GPU has CTA pairs, unequal numbers of key tiles; soft caps on both sides of
    the polynomial's range."""
    from teenygrad_b200 import ops
    B, H, S = 5, 12, 900
    parts = [planted(50 * b, S, H, H, D, V) for b in range(B)]
    q, k, v = (torch.cat([p[i] for p in parts]).to(BF) for i in range(3))
    gate, sink = (3 * rnd(7, B * S, H * V)).to(BF), torch.linspace(-3.0, 3.0, H)
    kc, vc = (t.view(B, S, H, -1).transpose(1, 2).contiguous().cuda() for t in (k, v))
    got = ops.cached_attention(q.cuda(), kc, vc, 0.15, entries_of([S] * B, range(B)), softcap=cap, sink=sink.cuda(), gate=gate.cuda()).double()
    g = om.sigmoid(gate.double()).view(-1, H, V)
    for b in range(B):
        s = slice(b * S, (b + 1) * S)
        want = om.causal_attention_fast(q[s].double(), k[s].double(), v[s].double(), 0.15, cap or None, sink.double()) * g[s]
        assert rel(got[s], want) < 1.5e-2, b


@DTYPES
@pytest.mark.parametrize("q_rank,rank,rot", [(72, 56, 24), (1536, 512, 64), (5000, 900, 8), (13, 21, 24), (40, 8, 0)])
def test_latent_norms_rotation_and_cache(dtype, q_rank, rank, rot):
    from teenygrad_b200 import ops
    pad = lambda n: (n + 7) // 8 * 8  # noqa: E731
    lens, pos, slots = [5, 1, 3], [0, 77, 3000], [1, 2, 0]
    rows, cap = sum(lens), 3004
    parts = [2 * rnd(1, rows, q_rank), 0.1 * rnd(2, rows, rank), rnd(3, rows, rot)]
    offs, proj = [], torch.zeros(rows, 0)
    for t in parts:
        offs.append(proj.shape[1])
        proj = torch.cat([proj, t, torch.zeros(rows, pad(t.shape[1]) - t.shape[1])], 1)
    proj = proj.to(dtype)
    qw, cw = 1 + 0.3 * rnd(4, q_rank), 1 + 0.3 * rnd(5, rank)
    freq, amp = om.rotation_frequencies(rot, 1000.0, om.yarn(2.0, 500)) if rot else ([], 1.0)
    cache = torch.full((3, cap, pad(rank) + rot), 7.0, dtype=dtype, device="cuda")
    latents = torch.zeros(rows, pad(rank) + rot, dtype=dtype, device="cuda")
    padded = lambda w: torch.nn.functional.pad(w, (0, pad(len(w)) - len(w))).cuda()  # noqa: E731
    table = entries_of(lens, slots, pos)
    cq = ops.latent_prepare(proj.cuda(), offs, q_rank, rank, padded(qw), padded(cw), torch.tensor(freq).float().cuda() if rot else None, 1e-3,
                            cache, ops.seq_table(table), max(lens), rot_scale=amp, latents=latents)
    x = proj.double()
    p = torch.cat([torch.arange(n) + s for n, s in zip(lens, pos)])
    tol = 3e-4 if dtype == F32 else 5e-3
    assert rel(cq[:, :q_rank], om.rms(x[:, :q_rank], 1e-3) * qw.double()) < tol and not cq[:, q_rank:].any()
    want = torch.zeros(rows, pad(rank) + rot, dtype=F64)
    want[:, :rank] = om.rms(x[:, offs[1]:offs[1] + rank], 1e-3) * cw.double()
    if rot:
        want[:, pad(rank):] = rotate_half(x[:, None, offs[2]:offs[2] + rot], p, freq, amp)[:, 0]
    assert rel(latents, want) < tol
    for slot, at, r0, n in table:
        assert torch.equal(cache[slot, at:at + n], latents[r0:r0 + n])
        cache[slot, at:at + n] = 7.0
    assert bool((cache == 7.0).all())


@DTYPES
@pytest.mark.parametrize("heads,n,k,rot", [(4, 88, 40, 24), (3, 512, 128, 64), (2, 128, 512, 0), (5, 8, 24, 8), (1, 40, 1024, 0)])
@pytest.mark.parametrize("lens", [[1, 1, 1], [5, 1, 12], [60, 33, 1]], ids=str)
def test_per_head_products(dtype, heads, n, k, rot, lens):
    from teenygrad_b200 import ops
    rows, pos = sum(lens), [7, 0, 900]
    x = rnd(1, rows, heads, rot + k).to(dtype)
    w = (rnd(2, heads, n, k) * k ** -0.5).to(dtype)
    freq, amp = om.rotation_frequencies(rot, 300.0, om.yarn(4.0, 100)) if rot else ([], 1.0)
    table = entries_of(lens, [0, 1, 2], pos)
    xd = x.cuda()
    out = ops.head_linear(xd[:, :, rot:], w.cuda(), rot, -rot, torch.tensor(freq).float().cuda() if rot else None, amp, ops.seq_table(table))
    want = torch.einsum("thk,hnk->thn", x[:, :, rot:].double(), w.double())
    assert rel(out[..., :n], want) < (1e-5 if dtype == F32 else 5e-3)
    if rot:
        p = torch.cat([torch.arange(m) + s for m, s in zip(lens, pos)])
        assert rel(out[..., n:], rotate_half(x[:, :, :rot].double(), p, freq, amp)) < (2e-4 if dtype == F32 else 5e-3)


@DTYPES
@pytest.mark.parametrize("heads,dim,vdim", [(4, 104, 88), (32, 576, 512), (8, 320, 256), (6, 72, 64), (3, 40, 24), (16, 192, 128), (2, 1000, 600), (5, 296, 256)])
@pytest.mark.parametrize("cuts", ["portions", "decode", "batch"])
def test_latent_attention(dtype, heads, dim, vdim, cuts):
    """One shared key per token; queries that single out a near, a far, the first or a border key."""
    from teenygrad_b200 import ops
    T, scale = 280, 0.2
    q, k, _ = (t.to(dtype) for t in planted(5, T, heads, 1, dim, 1))
    q = (q * (0.3 + 5.0 / dim ** 0.5)).to(dtype)
    want = om.causal_attention_fast(q.double(), k.double(), k[:, :, :vdim].double(), scale)
    cache = torch.full((3, 1024 if cuts == "decode" else T, dim), float("nan"), dtype=dtype, device="cuda")
    cache[1, :T] = k[:, 0].cuda()
    tol = 2e-5 if dtype == F32 else 1.5e-2
    if cuts == "batch":  # entries of one sequence at different places, in one step
        table = entries_of([1, 40, 1, 2, 17], [1] * 5, [279, 64, 0, 62, 127])
        rows = torch.cat([torch.arange(p, p + n) for _, p, _, n in table])
        got = ops.latent_attention(q[rows].cuda(), cache, vdim, scale, ops.seq_table(table), 40)
        assert rel(got, want[rows]) < tol
        return
    sizes = [2, 61, 1, 1, 3, 60, 5, 63, 64, 20] if cuts == "portions" else [1] * 5 + [59, 1, 1, 1, 1] + [1] * 212
    at, out = 0, []
    for n in sizes:
        out.append(ops.latent_attention(q[at:at + n].cuda(), cache, vdim, scale, ops.seq_table([(1, at, 0, n)]), n))
        at += n
    assert at == T and rel(torch.cat(out), want) < tol


# ------------------------------------------------------------------------------------------------ models
def config_a():
    """Odd sizes throughout: vocabulary, feed-forward, head counts, ranks and widths that no tile divides; a cap that bites."""
    return om.make_config(90, 131, [
        om.attention_layer(6, 3, 22, 10, 14, 900.0, 0.3, 4.0, True, ff=100), om.latent_layer(3, 18, 10, 14, 21, 27, 500.0, 0.35, om.yarn(4.0, 40, 8.0, 1.5)),
        om.attention_layer(3, 3, 20, 10, 20, 60.0, 0.4, 25.0, True), om.attention_layer(4, 1, 12, 20, 6, 1e4, 0.5, 9.0, False, ff=40),
        om.latent_layer(5, 12, 6, 8, 9, 13, 1e4, 0.5, None, ff=72), om.attention_layer(6, 3, 30, 10, 8, 100.0, 0.3, 15.0, True, ff=24)],
        eps=1e-4, mult=0.6, logit_scale=1.7)


def config_b():
    """Head sizes of the fast kernels: latents first and last, equal sizes everywhere else."""
    return om.make_config(128, 256, [
        om.latent_layer(4, 64, 32, 64, 128, 128, 1e4, 0.12, om.yarn(8.0, 128)), om.attention_layer(8, 2, 128, 128, 64, 1e4, 0.1, 30.0, True, ff=192),
        om.latent_layer(4, 128, 64, 128, 256, 512, 5e5, 0.07, om.yarn(40.0, 256)), om.attention_layer(8, 2, 128, 128, 128, 1e4, 0.1, 50.0, True),
        om.latent_layer(2, 96, 32, 96, 64, 256, 1e3, 0.1, None, ff=130)], mult=1.0, logit_scale=1.0)


def config_c():
    """No layer mixes values; one layer of each kind; everything equal or one."""
    return om.make_config(64, 64, [
        om.attention_layer(1, 1, 64, 64, 64, 1e4, 0.2, 8.0, False, ff=64), om.latent_layer(1, 64, 64, 64, 64, 64, 1e4, 0.15, om.yarn(1.0, 64), ff=64)],
        mult=1.0, logit_scale=1.0)


def peaked(cfg, seed):
    """Random weights whose attention is decided by single keys."""
    w = om.make_weights(cfg, seed)
    for name in w:
        if name.endswith(("mix.q", "mix.uq")):
            w[name] = (w[name].float() * 3).to(BF)
    return w


CASES = {"a": (config_a, (5, 90, 201, 330)), "b": (config_b, (5, 90, 201, 330)), "c": (config_c, (5, 90, 201, 330))}
_cache = {}


def case(name):
    if name not in _cache:
        make, lens = CASES[name]
        cfg = make()
        w = peaked(cfg, 7)
        toks = {n: torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(n)).tolist() for n in lens}
        _cache[name] = cfg, w, toks, {n: om.forward(cfg, w, t) for n, t in toks.items()}
    return _cache[name]


def build(name, dtype, **kw):
    from teenygrad_b200 import molitar
    cfg, w, _, _ = case(name)
    return molitar.build(cfg, w, dtype, **{"max_batch": 4, "max_len": 400, "max_rows": 400, **kw})


def close(got, want, dtype):
    """f32: every logit; bf16: rms error of every position."""
    d = got.double().cpu() - want
    scale = float(want.pow(2).mean().sqrt())
    if dtype == F32:
        assert float(d.abs().max()) < 5e-4 * scale
    else:
        assert float(d.pow(2).mean(-1).sqrt().max()) < 0.12 * scale and float(d.pow(2).mean().sqrt()) < 0.04 * scale


MODELS = pytest.mark.parametrize("name", sorted(CASES))


@MODELS
@DTYPES
def test_whole_prompts(name, dtype):
    r = build(name, dtype)
    _, _, toks, want = case(name)
    for n, t in toks.items():
        s = r.open()
        close(r.step([(s, t, range(n))])[0], want[n], dtype)
        r.close(s)


@MODELS
@DTYPES
@pytest.mark.parametrize("sizes", [[2], [3, 17, 1, 40], [64], [1, 31, 2, 16, 100], [130, 63, 65]], ids=str)
def test_portions_and_token_by_token(name, dtype, sizes):
    """A prompt cut anywhere, its last tokens one by one; the slot has held another sequence before."""
    r = build(name, dtype, max_batch=1)
    _, _, toks, want = case(name)
    s = r.open()
    r.step([(s, toks[330], [])])
    r.close(s)
    s, t, at, i, out = r.open(), toks[201], 0, 0, []
    while at < len(t):
        n = min(sizes[i % len(sizes)], len(t) - at) if at < 150 else 1
        out += r.step([(s, t[at:at + n], range(n))])
        at, i = at + n, i + 1
    close(torch.cat(out), want[201], dtype)


@MODELS
@DTYPES
def test_unequal_batches_equal_each_alone(name, dtype):
    """Prefills, portions and single tokens of several requests mixed in one step; steps larger than the workspace are split."""
    r = build(name, dtype, max_tokens=250, max_rows=120)
    _, _, toks, want = case(name)
    seqs = {n: r.open() for n in (330, 5, 90)}
    at = {n: 0 for n in seqs}
    got = {n: [] for n in seqs}
    plan = [{330: 200, 5: 2}, {330: 1, 90: 50, 5: 1}, {5: 2, 90: 1, 330: 100}, {90: 39, 330: 29}]
    for step in plan:
        entries = [(seqs[n], toks[n][at[n]:at[n] + c], range(c)) for n, c in step.items()]
        for n, o in zip(step, r.step(entries)):
            got[n].append(o)
            at[n] += step[n]
    for n in seqs:
        close(torch.cat(got[n]), want[n], dtype)
    # slots in another order, freed and used again
    for n in (90, 330):
        r.close(seqs[n])
    again = {90: r.open(), 201: r.open()}
    o90, o201 = r.step([(again[90], toks[90], range(90)), (again[201], toks[201], range(201))])
    close(o90, want[90], dtype)
    close(o201, want[201], dtype)


@MODELS
@DTYPES
def test_batches_of_whole_prompts(name, dtype):
    """Several fresh prompts in one step: equal ones (one attention launch), then unequal ones behind a running sequence."""
    r = build(name, dtype, max_tokens=1000, max_rows=1000)
    _, _, toks, want = case(name)
    seqs = [r.open() for _ in range(3)]
    for o in r.step([(s, toks[201], range(201)) for s in seqs]):
        close(o, want[201], dtype)
    for s in seqs[1:]:
        r.close(s)
    r.close(seqs[0])
    live = r.open()
    r.step([(live, toks[330][:300], [])])
    more = [r.open() for _ in range(3)]
    outs = r.step([(live, toks[330][300:], range(30)), (more[0], toks[201], range(201)), (more[1], toks[90], range(90)), (more[2], toks[5], range(5))])
    for o, w in zip(outs, (want[330][300:], want[201], want[90], want[5])):
        close(o, w, dtype)


@MODELS
@DTYPES
def test_layers_one_by_one(name, dtype):
    """Residual stream after every prefix of the layers."""
    from teenygrad_b200 import molitar
    cfg, w, toks, _ = case(name)
    _, layers = om.forward(cfg, w, toks[90], want_layers=True)
    for n in range(1, len(cfg["layers"]) + 1):
        r = molitar.build({**cfg, "layers": cfg["layers"][:n]}, w, dtype, max_batch=1, max_len=100)
        r.step([(r.open(), toks[90], [0])])
        got = r.residual_stream().double().cpu()
        d = (got - layers[n - 1]).pow(2).mean().sqrt() / layers[n - 1].pow(2).mean().sqrt()
        assert float(d) < (1e-5 if dtype == F32 else 2e-2), n


@MODELS
def test_greedy_generation_follows_the_oracle(name):
    """f32: the generated ids are the oracle's, through graph replay and without; batches of unequal prompts, groups."""
    cfg, w, toks, _ = case(name)
    r = build(name, F32, max_new_tokens=24)
    prompts = [toks[5], toks[90], toks[201]]
    ids = r.generate(prompts, 24).cpu()
    assert torch.equal(ids, r.generate(prompts, 24, use_graph=False).cpu())
    for p, row in zip(prompts, ids.tolist()):
        logits = om.forward(cfg, w, p + row[:-1])[len(p) - 1:]
        top = logits.topk(2).values
        best = logits.argmax(-1).tolist()
        for i, (a, b) in enumerate(zip(row, best)):
            assert a == b or float(top[i, 0] - logits[i, a]) < 1e-3, i
    many = r.generate([toks[5], toks[5][:3], toks[90], toks[5], toks[90], toks[5]], 6).cpu()  # more than there are slots
    assert torch.equal(many[0], many[3]) and torch.equal(many[2], many[4]) and torch.equal(many[2], ids[1, :6])
    assert len(r._free) == r.max_batch


@MODELS
def test_bf16_generation_graph_batch_and_long_decoding(name):
    """A long decode by graph replay: its logits at the end equal those of the whole text at once."""
    r = build(name, BF, max_new_tokens=200)
    _, _, toks, _ = case(name)
    p = torch.tensor([toks[90], toks[201][:90]], dtype=torch.int32)
    ids = r.generate(p, 200)
    last = r.logits().float().clone()
    ids = ids.cpu().tolist()
    for b in range(2):
        s = r.open()
        text = p[b].tolist() + ids[b][:-1]
        whole = r.step([(s, text, [len(text) - 1])])[0]
        r.close(s)
        d = (last[b] - whole[0]).pow(2).mean().sqrt() / whole.pow(2).mean().sqrt()
        assert float(d) < 0.1
    r.set_sampling(0.8, top_k=20, seed=5)
    a, b = r.generate(p, 16).cpu(), r.generate(p, 16, use_graph=False).cpu()
    assert torch.equal(a, b)


def test_first_tokens_of_a_sequence():
    """Single-token requests, and prompts whose first portion is one token."""
    cfg, w, toks, want = case("a")
    for dtype in (F32, BF):
        r = build("a", dtype)
        seqs = [r.open() for _ in range(3)]
        outs = r.step([(s, toks[n][:1], [0]) for s, n in zip(seqs, (5, 90, 330))])
        for o, n in zip(outs, (5, 90, 330)):
            close(o, want[n][:1], dtype)
        outs = r.step([(s, toks[n][1:3], [0, 1]) for s, n in zip(seqs, (5, 90, 330))])
        for o, n in zip(outs, (5, 90, 330)):
            close(o, want[n][1:3], dtype)


@DTYPES
@pytest.mark.parametrize("n", [1, 2, 9, 63, 65, 129])
def test_capacity_of_exactly_the_sequence(dtype, n):
    """A runner that holds no token more than the request, at once and token by token."""
    cfg, w, toks, want = case("b")
    r = build("b", dtype, max_batch=1, max_len=n, max_rows=n)
    for sizes in ([n], [1] * n):
        s, at, out = r.open(), 0, []
        for c in sizes:
            out += r.step([(s, toks[201][at:at + c], range(c))])
            at += c
        r.close(s)
        close(torch.cat(out), want[201][:n], dtype)


def test_command_line_and_trace_replay(tmp_path):
    from teenygrad_b200 import safetensors
    cfg, w, toks, want = case("a")
    safetensors.save_file(w, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    t = toks[90]
    out = subprocess.run([sys.executable, "-m", "teenygrad_b200.generate", "--model", str(tmp_path), "--dtype", "float32", "--prompt",
                          ",".join(map(str, toks[5])), "--prompt", ",".join(map(str, t)), "--max-new-tokens", "3"],
                         cwd=ROOT, capture_output=True, text=True, timeout=300, check=True)
    lines = [[int(x) for x in ln.split(",")] for ln in out.stdout.split()]
    assert [ln[0] for ln in lines] == [int(want[5][-1].argmax()), int(want[90][-1].argmax())]
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": t[:50], "want": [3, 49]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": t[50:52], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": t[52:], "want": [37, 0]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": toks[5], "want": [4]}], "end": ["y"]}]
    out = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path),
                          "--max-tokens", "95"], input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=300, check=True)
    assert [ln for ln in out.stdout.split("\n") if ln.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    for n, places in ((0, [want[90][3], want[90][49]]), (2, [want[90][89], want[90][52]]), (3, [want[5][4]])):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{n}.f32", dtype="<f4")).view(-1, cfg["vocab"])
        close(got, torch.stack(places), F32)
    assert not (tmp_path / "1.f32").exists()
