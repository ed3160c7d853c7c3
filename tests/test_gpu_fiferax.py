"""The Fiferax decoder and the hybrid runner on a GPU, against the plain float64 restatement in oracle/fiferax.py: every
mechanism alone (through its own entry point), whole prompts, portions, token-by-token decoding, unequal batches, reused
slots, and generation through the runner, the command line and the trace replay."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import fiferax as of

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


# ------------------------------------------------------------------------------------------------ mechanisms alone
@DTYPES
@pytest.mark.parametrize("heads,dim", [(3, 64), (2, 128), (2, 40), (1, 200), (3, 22), (2, 9)])
def test_delta_rule(dtype, heads, dim):
    """Unequal entries from fresh slots, then a second step that carries the states on (and leaves a slot alone)."""
    from teenygrad_b200 import ops
    n = heads * dim
    lens1, slots, lens2 = [37, 1, 90], [2, 0, 3], [3, 50, 16]
    state = torch.full((5, heads, dim, dim), 7.0, device="cuda")  # fresh entries must not read what a slot holds
    w_bias, a_bias = rnd(1, n), rnd(2, n)
    cu = {s: None for s in slots}
    for step, lens in enumerate((lens1, lens2)):
        rows = sum(lens)
        proj = rnd(10 + step, rows, 4 * n + 6).to(dtype)
        wz = (2 * rnd(20 + step, rows, n)).to(dtype)
        pos = [0, 0, 0] if step == 0 else lens1
        table = entries_of(lens, slots, pos)
        o = ops.state_scan_delta(proj.cuda(), (0, n, 2 * n, 3 * n), wz.cuda(), w_bias.cuda(), a_bias.cuda(), 0.6, 1e-6, state,
                                 ops.seq_table(table), max(lens))
        for slot, _, r0, ln in table:
            p = proj[r0:r0 + ln].double()
            r, k, v, a = (p[:, i * n:(i + 1) * n].view(ln, heads, dim) for i in range(4))
            w = torch.exp(-0.6 * of.sigmoid(wz[r0:r0 + ln].double() + w_bias.double())).view(ln, heads, dim)
            a = of.sigmoid(a + a_bias.double().view(heads, dim))
            want, cu[slot] = of.delta_recurrence(r, k, v, w, a, cu[slot])
            tol = 1e-5 if dtype == F32 else 1e-4
            assert rel(o[r0:r0 + ln], want.reshape(ln, n)) < tol, (step, slot)
            assert rel(state[slot], cu[slot]) < tol, (step, slot)
    assert bool((state[1] == 7.0).all()) and bool((state[4] == 7.0).all())


@DTYPES
@pytest.mark.parametrize("heads,dk,dv", [(3, 64, 64), (2, 128, 128), (2, 40, 72), (2, 128, 160), (1, 18, 33), (1, 7, 260), (2, 256, 24)])
def test_scalar_decay_state(dtype, heads, dk, dv):
    from teenygrad_b200 import ops
    decay = torch.tensor([0.999, 0.01, 0.8][:heads])  # one that forgets within a token or two: no division by its powers
    offs = (0, heads * dk, 2 * heads * dk)
    state = torch.zeros(2, heads, dk, dv, device="cuda")
    S = None
    for step, ln in enumerate((70, 1, 1, 33, 2)):
        proj = rnd(step, ln, heads * (2 * dk + dv)).to(dtype)
        o = ops.state_scan_decay(proj.cuda(), offs, decay.cuda(), state, ops.seq_table([(1, sum((70, 1, 1, 33, 2)[:step]), 0, ln)]), ln)
        q, k, v = of.silu(proj.double()).split([heads * dk, heads * dk, heads * dv], 1)
        want, S = of.decay_recurrence(q.view(ln, heads, dk), k.view(ln, heads, dk), v.view(ln, heads, dv), decay.double(), S)
        tol = 1e-5 if dtype == F32 else 2e-2  # the activated projections are bf16 tensors
        assert rel(o, want.reshape(ln, heads * dv)) < tol and rel(state[1], S) < tol, step


@DTYPES
@pytest.mark.parametrize("width", [64, 129, 30])
def test_minimal_gru(dtype, width):
    from teenygrad_b200 import ops
    zb, xb = rnd(1, width), torch.zeros(width)
    state = torch.full((3, width), 9.0, device="cuda")
    S = {2: None, 0: None}
    for step, lens in enumerate(([200, 5], [1, 1], [17, 300])):
        pos = [0, 0] if step == 0 else [200 + step, 5 + step]
        table = entries_of(lens, [2, 0], pos)
        proj = rnd(5 + step, sum(lens), 3 * width)
        proj[:, width:2 * width][::3] = 0.0     # the branch point of the candidate
        proj = proj.to(dtype)
        out = ops.min_gru(proj.cuda(), (0, width, 2 * width), zb.cuda(), xb.cuda(), state, ops.seq_table(table), max(lens), scale=1.5)
        for slot, _, r0, ln in table:
            z, u, g = proj[r0:r0 + ln].double().split(width, 1)
            h, S[slot] = of.min_gru(z + zb.double(), u, S[slot])
            assert rel(out[r0:r0 + ln], 1.5 * h * of.silu(g)) < (1e-5 if dtype == F32 else 1e-2)
            assert rel(state[slot], S[slot]) < 1e-5
    assert bool((state[1] == 9.0).all())


@DTYPES
@pytest.mark.parametrize("cols,group", [(192, 64), (256, 128), (96, 32), (4096, 4096), (120, 120), (90, 30), (77, 11)])
def test_gated_group_norm(dtype, cols, group):
    from teenygrad_b200 import ops
    o, gate, w = 3 * rnd(1, 19, cols), rnd(2, 19, cols).to(dtype), rnd(3, cols)
    got = ops.gated_rms_norm(o.cuda(), gate.cuda(), w.cuda(), group, 1e-3, scale=0.7)
    want = 0.7 * of.rms_norm(o.double().view(19, -1, group), 1.0, 1e-3).view(19, cols) * w.double() * of.sigmoid(gate.double())
    assert rel(got, want) < (1e-5 if dtype == F32 else 5e-3)


@DTYPES
@pytest.mark.parametrize("heads,kv,dim,rot", [(4, 2, 64, 32), (3, 1, 128, 128), (2, 2, 20, 6), (5, 5, 96, 96), (2, 1, 80, 0)])
def test_head_norm_and_rotary(dtype, heads, kv, dim, rot):
    from teenygrad_b200 import ops
    lens, pos = [9, 4], [0, 1900]
    rows = sum(lens)
    qkv = (3 * rnd(1, rows, heads + kv, dim)).to(dtype).cuda()
    q, k = qkv[:, :heads].clone(), qkv[:, heads:]
    qw, kw = 1 + 0.3 * rnd(2, dim), 1 + 0.3 * rnd(3, dim)
    base = 700.0
    inv = (base ** (torch.arange(rot // 2, dtype=F64) * (-2.0 / max(rot, 1)))).float()
    got_k = ops.head_norm_rope(q, k, qw.cuda(), kw.cuda(), inv.cuda() if rot else None, rot, 1e-4, ops.seq_table(entries_of(lens, [0, 1], pos)),
                               max(lens))
    p = torch.cat([torch.arange(n) + s for n, s in zip(lens, pos)])
    x = qkv.double().cpu()
    for got, src, w in ((q, x[:, :heads], qw), (got_k, x[:, heads:], kw)):
        assert rel(got, of.rotary_half(of.rms_norm(src, w.double(), 1e-4), p, rot, base)) < (2e-4 if dtype == F32 else 5e-3)


def planted(seed, T, heads, kv, dim, window):
    """Random queries and keys in which some queries match one key so well that it takes all the weight if it is visible: keys
    at the window's edge (just inside, just outside), one token away and far away."""
    q, k = rnd(seed, T, heads, dim), rnd(seed + 1, T, kv, dim)
    v = rnd(seed + 2, T, kv, dim)
    for n, i in enumerate(range(5, T, 7)):
        j = i - (window - 1, window, 1, 0, window // 2)[n % 5]
        if 0 <= j < T:
            q[i] = 4.0 * k[j].repeat_interleave(heads // kv, 0)
    return q, k, v


@DTYPES
@pytest.mark.parametrize("heads,kv,dim,window", [(4, 1, 128, 130), (2, 2, 128, 64), (4, 2, 64, 33), (3, 1, 80, 50), (2, 1, 136, 20), (2, 2, 20, 9),
                                                 (2, 1, 128, 1), (2, 1, 64, 1000), (8, 1, 64, 70)])
@pytest.mark.parametrize("cuts", ["whole", "uniform", "portions", "decode"])
def test_windowed_attention(dtype, heads, kv, dim, window, cuts):
    from teenygrad_b200 import ops
    T = 300
    q, k, v = (t.to(dtype) for t in planted(3, T, heads, kv, dim, window))
    want = of.window_attention_fast(q.double(), k.double(), v.double(), 0.3, window) * 0.8
    ring = min(window, T)
    rings = [torch.full((3, kv, ring, dim), float("nan"), dtype=dtype, device="cuda") for _ in range(2)]
    qd, kd, vd = (t.cuda() for t in (q, k, v))
    sizes = {"whole": [T], "uniform": [T], "portions": [2, 63, 64, 1, 65, 3, 2, 100], "decode": [T - 70] + [1] * 70}[cuts]
    at, out = 0, []
    for n in sizes:
        s = slice(at, at + n)
        out.append(ops.window_attention(qd[s], kd[s], vd[s], *rings, window, 0.3, ops.seq_table([(1, at, 0, n)]), n, out_scale=0.8,
                                        uniform_fresh=cuts == "uniform"))
        at += n
    got = torch.cat(out)
    assert rel(got, want) < (2e-5 if dtype == F32 else 1.5e-2)


def test_windowed_attention_uniform_batch():
    """Whole prompts of one length, head size 128, several query tiles and windows around the tile sizes."""
    from teenygrad_b200 import ops
    B, T, H, G, D = 3, 700, 4, 2, 128
    for window in (100, 128, 129, 256, 300, 699, 5000):
        parts = [planted(10 * b + window, T, H, G, D, window) for b in range(B)]
        q, k, v = (torch.cat([p[i] for p in parts]).to(BF) for i in range(3))
        rings = [torch.zeros(B, G, min(window, T), D, dtype=BF, device="cuda") for _ in range(2)]
        got = ops.window_attention(q.cuda(), k.cuda(), v.cuda(), *rings, window, 0.1, ops.seq_table(entries_of([T] * B, range(B))), T, uniform_fresh=True)
        for b in range(B):
            s = slice(b * T, (b + 1) * T)
            assert rel(got[s], of.window_attention_fast(q[s].double(), k[s].double(), v[s].double(), 0.1, window)) < 1.5e-2, (window, b)


@DTYPES
@pytest.mark.parametrize("n", [96, 4096, 50])
def test_residual_norm(dtype, n):
    from teenygrad_b200 import ops
    x, d, w = 5 * rnd(1, 33, n), rnd(2, 33, n).to(dtype), rnd(3, n)
    xd = x.cuda()
    y = ops.residual_rms_norm(xd, d.cuda(), w.cuda(), 1e-2)
    s = x.double() + d.double()
    assert rel(xd, s) < 1e-6 and rel(y, of.rms_norm(s, w.double(), 1e-2)) < (1e-5 if dtype == F32 else 5e-3)


# ------------------------------------------------------------------------------------------------ models
def config_a():
    """Odd sizes throughout: vocabulary, feed-forward, head counts and widths that no tile divides."""
    return of.make_config(96, 133, [
        of.gru_layer(40, ff=100), of.parallel_layer(6, 3, 32, 9, 16, 5000.0, 0.3, 3, 24, 40, [0.5, 0.9, 0.97], 0.7, 1.3, ff=72),
        of.delta_layer(3, 32), of.parallel_layer(3, 3, 20, 40, 20, 300.0, 0.5, 1, 8, 12, [0.99], 1.1, 0.6), of.delta_layer(1, 64, ff=64)],
        eps=1e-4, scale=1.7)


def config_b():
    """Head sizes of the fast kernels."""
    return of.make_config(128, 257, [
        of.delta_layer(2, 64, ff=192), of.parallel_layer(4, 1, 128, 150, 64, 10000.0, 0.2, 2, 64, 96, [0.7, 0.995], 1.0, 1.0, ff=130),
        of.gru_layer(200), of.parallel_layer(4, 2, 64, 33, 64, 1000.0, 0.25, 1, 128, 128, [0.98], 0.5, 1.5)], scale=1.0)


def peaked(cfg, seed, rank):
    """Random weights whose attention is decided by single keys."""
    w = of.make_weights(cfg, seed, rank)
    for name in w:
        if name.endswith("q.norm"):
            w[name] = (w[name].float() * 3).to(BF)
    return w


CASES = {"a": (config_a, 5), "b": (config_b, 16)}
_cache = {}


def case(name):
    if name not in _cache:
        make, rank = CASES[name]
        cfg = make()
        w = peaked(cfg, 7, rank)
        toks = {n: torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(n)).tolist() for n in (5, 90, 201, 330)}
        _cache[name] = cfg, w, toks, {n: of.forward(cfg, w, t) for n, t in toks.items()}
    return _cache[name]


def build(name, dtype, **kw):
    from teenygrad_b200 import fiferax
    cfg, w, _, _ = case(name)
    return fiferax.build(cfg, w, dtype, **{"max_batch": 4, "max_len": 400, "max_rows": 400, **kw})


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
@pytest.mark.parametrize("sizes", [[2], [3, 17, 1, 40], [64], [1, 31, 2, 16, 100]], ids=str)
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
    r = build(name, dtype, max_tokens=128, max_rows=60)
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
def test_layers_one_by_one(name, dtype):
    """Residual stream after every prefix of the layers."""
    from teenygrad_b200 import fiferax
    cfg, w, toks, _ = case(name)
    _, layers = of.forward(cfg, w, toks[90], want_layers=True)
    for n in range(1, len(cfg["layers"]) + 1):
        r = fiferax.build({**cfg, "layers": cfg["layers"][:n]}, w, dtype, max_batch=1, max_len=100)
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
        logits = of.forward(cfg, w, p + row[:-1])[len(p) - 1:]
        top = logits.topk(2).values
        best = logits.argmax(-1).tolist()
        for i, (a, b) in enumerate(zip(row, best)):
            assert a == b or float(top[i, 0] - logits[i, a]) < 1e-3, i
    many = r.generate([toks[5], toks[5][:3], toks[90], toks[5], toks[90], toks[5]], 6).cpu()  # more than there are slots
    assert torch.equal(many[0], many[3]) and torch.equal(many[2], many[4]) and torch.equal(many[2], ids[1, :6])
    assert len(r._free) == r.max_batch


@MODELS
def test_bf16_generation_graph_batch_and_long_decoding(name):
    """A long decode (well past every window) by graph replay: its logits at the end equal those of the whole text at once."""
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


def test_bad_steps_are_refused():
    from teenygrad_b200._lib import TeenyError
    r = build("a", BF, max_batch=2, max_len=20)
    s = r.open()
    with pytest.raises(ValueError, match="max_len"):
        r.step([(s, [1] * 21, [])])
    with pytest.raises(ValueError, match="vocabulary"):
        r.step([(s, [133], [])])
    with pytest.raises(TeenyError):
        r._run(torch.zeros(2, dtype=torch.int32, device="cuda"), [s, s], [1, 1], [])  # one slot twice
    r.open()
    with pytest.raises(RuntimeError, match="slots"):
        r.open()


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
