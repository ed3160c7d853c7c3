"""Hybrid decoder runner: host wrapper over the C++ executor of include/teeny_hybrid.h.

``HybridConfig`` describes a decoder as layers of parallel branches (windowed, full or latent attention, delta rule,
scalar-decay state, minimal GRU) and an optional gated feed-forward; a design's own module turns its config.json into one and hands
the weights over layer by layer (``HybridRunner.load_layer``).  Sequences live in state slots: ``open`` / ``step`` /
``close`` feed any tokens of any sequences, ``generate`` runs whole prompts and decodes with CUDA-graph replay.
"""
import ctypes as C
import math
from dataclasses import dataclass, field

import torch

from . import _lib
from ._lib import lib, check, vp, i32, f32, sz
from .runner import BUF_LOGITS, DecoderRunner, stream

ATTENTION, DELTA, DECAY, MIN_GRU, LATENT = range(5)
QK_NORM, KEYS_ARE_VALUES, SINK, OUT_GATE, VALUE_MIX = 1, 2, 4, 8, 16
IN_BIAS, POST_NORM = 1, 2  # layer flags
ACT_SILU, ACT_GELU_TANH = 1, 2

W_NORM1, W_NORM2, W_IN, W_OUT, W_GATE_UP, W_DOWN, W_IN_BIAS, W_NORM1_POST, W_NORM2_POST = range(9)
BRANCH_VECTORS = {"q_norm": 50, "k_norm": 51, "o_norm": 52, "decay_bias": 54, "rate_bias": 55, "z_bias": 56, "x_bias": 57,
                  "decay": 58, "inv_freq": 59, "sink": 60, "value_mix": 61}
W_LOW, W_UQ, W_EXPAND, W_ABSORB, W_VALUE_UP = 53, 62, 63, 64, 65
W_EMBED, W_FINAL_NORM, W_LM_HEAD = 100, 101, 102
BUF_RESIDUAL, BUF_LAST_DELTA = 4, 5


class _Cfg(C.Structure):
    """teeny_hybrid_config"""
    _fields_ = [(n, i32) for n in ("num_layers", "num_branches", "width", "vocab")] + [("eps", f32), ("embed_scale", f32), ("residual_mult", f32)] + \
               [(n, i32) for n in ("f32", "max_batch", "max_len", "max_tokens", "max_rows", "max_new_tokens")]


class _Layer(C.Structure):
    """teeny_hybrid_layer"""
    _fields_ = [(n, i32) for n in ("first_branch", "num_branches", "ff", "act", "flags")]


class _Branch(C.Structure):
    """teeny_hybrid_branch"""
    _fields_ = [(n, i32) for n in ("kind", "heads", "kv_heads", "dim", "vdim", "rank", "q_rank", "window", "rot_dims", "flags")] + \
               [(n, f32) for n in ("score_scale", "out_scale", "decay_coef", "unit_eps", "softcap", "rot_scale")]


_P = C.POINTER
_DESC = [_P(_Cfg), _P(_Layer), _P(_Branch)]
SIGNATURES = {
    "teeny_hybrid_workspace_bytes": (sz, _DESC),
    "teeny_hybrid_slot_bytes": (sz, _DESC),
    "teeny_hybrid_create": (i32, _DESC + [vp, sz, vp, _P(vp)]),
    "teeny_hybrid_destroy": (None, [vp]),
    "teeny_hybrid_set_weight": (i32, [vp, i32, i32, i32, vp]),
    "teeny_hybrid_step": (i32, [vp, vp, _P(i32), _P(i32), _P(i32), i32, _P(i32), i32, vp]),
    "teeny_hybrid_begin": (i32, [vp, vp]),
    "teeny_hybrid_decode": (i32, [vp, vp]),
    "teeny_hybrid_set_sampling": (i32, [vp, f32, i32, f32, C.c_ulonglong]),
    "teeny_hybrid_capture_decode": (i32, [vp, vp]),
    "teeny_hybrid_decode_replay": (i32, [vp, vp]),
    "teeny_hybrid_buffer": (vp, [vp, i32]),
}
_lib.bind(SIGNATURES)


@dataclass
class Branch:
    kind: int
    dim: int
    heads: int = 1
    kv_heads: int = 0
    vdim: int = 0
    rank: int = 0
    q_rank: int = 0
    window: int = 0          # attention: 0 = every earlier token
    rot_dims: int = 0
    rot_base: float = 10000.0
    inv_freq: list = None    # angle per position of every rotated pair, where it is not rot_base^(-2 i / rot_dims)
    rot_scale: float = 1.0   # factor of cos and sin
    flags: int = 0
    score_scale: float = 1.0
    out_scale: float = 1.0
    decay_coef: float = 0.0
    unit_eps: float = 0.0
    softcap: float = 0.0
    decay: tuple = ()  # per head, for DECAY

    def input_sizes(self):
        """Rows of the parts of the fused input projection, in order (include/teeny_hybrid.h)."""
        n, nv = self.heads * self.dim, self.heads * self.vdim
        if self.kind == ATTENTION:
            k = self.kv_heads * self.dim
            return [n, k] + ([] if self.flags & KEYS_ARE_VALUES else [self.kv_heads * self.vdim]) + ([nv] if self.flags & OUT_GATE else [])
        if self.kind == LATENT:
            return [self.q_rank, self.rank, self.rot_dims]
        if self.kind == DELTA:
            return [n] * 5 + [self.rank]
        if self.kind == DECAY:
            return [n, n, nv, nv]
        return [self.dim] * 3

    def output_size(self):
        return self.dim if self.kind == MIN_GRU else self.heads * self.vdim

    def frequencies(self):
        if self.inv_freq is not None:
            return self.inv_freq
        return [float(self.rot_base) ** (-2.0 * i / self.rot_dims) for i in range(self.rot_dims // 2)]


@dataclass
class Layer:
    branches: list
    ff: int = 0
    act: int = 0
    flags: int = 0


@dataclass
class HybridConfig:
    width: int
    vocab: int
    eps: float
    embed_scale: float
    layers: list = field(default_factory=list)
    residual_mult: float = 1.0
    logit_scale: float = 1.0


@dataclass
class Sequence:
    """A live request: its state slot and how many of its tokens have been run."""
    slot: int
    pos: int = 0


def pad_to(n, m):
    return (n + m - 1) // m * m


def fuse_rows(parts, dtype):
    """Matrices stacked with every part starting at a multiple of 8 rows, rows padded to a multiple of 8 columns."""
    k = parts[0].shape[1]
    out = torch.zeros(sum(pad_to(p.shape[0], 8) for p in parts), pad_to(k, 8), dtype=dtype, device=parts[0].device)
    r = 0
    for p in parts:
        out[r:r + p.shape[0], :k] = p
        r += pad_to(p.shape[0], 8)
    return out


def fuse_columns(parts, dtype):
    """Matrices side by side with every part starting at a multiple of 8 columns."""
    out = torch.zeros(parts[0].shape[0], sum(pad_to(p.shape[1], 8) for p in parts), dtype=dtype, device=parts[0].device)
    c = 0
    for p in parts:
        out[:, c:c + p.shape[1]] = p
        c += pad_to(p.shape[1], 8)
    return out


def interleave_glu(gate, up, dtype):
    """Gate and up rows in alternating blocks of 64, zero rows beyond the feed-forward size; columns padded to 8."""
    ff, k = gate.shape
    f = pad_to(ff, 64)
    both = torch.zeros(2, f, pad_to(k, 8), dtype=dtype, device=gate.device)
    both[0, :ff, :k], both[1, :ff, :k] = gate, up
    return both.view(2, f // 64, 64, -1).transpose(0, 1).reshape(2 * f, -1).contiguous()


def pad_columns(w, multiple, dtype):
    out = torch.zeros(w.shape[0], pad_to(w.shape[1], multiple), dtype=dtype, device=w.device)
    out[:, :w.shape[1]] = w
    return out


def yarn_frequencies(dims, base, factor, original, fast, slow):
    """Rotary frequencies stretched to a longer context (YaRN): pairs with more than ``fast`` turns over the ``original``
    context stay, those with fewer than ``slow`` are divided by ``factor``, a linear ramp over the pair index joins them.
    Returns (frequencies, factor of cos and sin)."""
    def pair(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(pair(fast)), 0), min(math.ceil(pair(slow)), dims - 1)
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


@dataclass
class HeadRows:
    """How a checkpoint's head of ``dim`` rows, of which the first ``rot`` are rotated in neighbouring pairs (2 i, 2 i + 1),
    lies in the runner: first all even ones of the pairs, then all odd ones (the kernels rotate i with i + half), each padded
    to a multiple of 8 with zero rows, then the rest padded to a multiple of 8.  Query and key rows move alike, so scores stay
    the same; a padded pair is zero and gets frequency 0."""
    dim: int
    rot: int = 0

    @property
    def rot_rows(self):
        return 2 * pad_to(self.rot // 2, 8)

    @property
    def rows(self):
        return self.rot_rows + pad_to(self.dim - self.rot, 8)

    def place(self, w):
        """Rows (or elements) of any number of heads, [heads * dim, ...] -> [heads * rows, ...]."""
        w = w.reshape(-1, self.dim, *w.shape[1:])
        out = torch.zeros(w.shape[0], self.rows, *w.shape[2:], dtype=w.dtype, device=w.device)
        h, p = self.rot // 2, self.rot_rows // 2
        out[:, :h], out[:, p:p + h] = w[:, 0:self.rot:2], w[:, 1:self.rot:2]
        out[:, 2 * p:2 * p + self.dim - self.rot] = w[:, self.rot:]
        return out.reshape(-1, *w.shape[2:])

    def pad_frequencies(self, freq):
        return list(freq) + [0.0] * (self.rot_rows // 2 - len(freq))


def latent_weights(branch, uk, uv, dtype):
    """The per-head key and value projections of a latent attention branch, ``uk`` [heads * dim, rank] and ``uv`` [heads * vdim,
    rank], as the runner reads them: (EXPAND, ABSORB, VALUE_UP) of include/teeny_hybrid.h."""
    H, D, V, R, RD = branch.heads, branch.dim, branch.vdim, branch.rank, branch.rot_dims
    KR = pad_to(R, 8)
    expand = torch.zeros(H * (RD + D + V), KR + RD, dtype=dtype, device=uk.device)
    keys = expand[:H * (RD + D)].view(H, RD + D, KR + RD)
    keys[:, :RD, KR:] = torch.eye(RD, dtype=dtype, device=uk.device)  # the shared rotated part, copied to every head
    keys[:, RD:, :R] = uk.view(H, D, R)
    expand[H * (RD + D):, :R] = uv
    absorb = torch.zeros(H, KR, D, dtype=dtype, device=uk.device)
    absorb[:, :R] = uk.view(H, D, R).transpose(1, 2)
    up = torch.zeros(H, V, KR, dtype=dtype, device=uk.device)
    up[:, :, :R] = uv.view(H, V, R)
    return expand, absorb, up


def plan_steps(entries, max_tokens, max_rows):
    """Cuts entries (length, wanted places in ascending order) into steps of at most ``max_tokens`` tokens and
    ``max_rows`` wanted rows: yields lists of (entry, first, count, wanted places in [first, first + count)).  An entry's
    portions come in order, one per step."""
    step, tokens, rows = [], 0, 0
    for e, (n, want) in enumerate(entries):
        at, w = 0, 0
        while at < n:
            if tokens == max_tokens or rows == max_rows or (step and step[-1][0] == e):
                yield step
                step, tokens, rows = [], 0, 0
            count = min(n - at, max_tokens - tokens)
            here = [p for p in want[w:] if p < at + count]
            if rows + len(here) > max_rows:  # stop in front of the first place that has no row left
                here = here[:max_rows - rows]
                count = want[w + len(here)] - at
                if count == 0:
                    yield step
                    step, tokens, rows = [], 0, 0
                    continue
            step.append((e, at, count, here))
            at, w, tokens, rows = at + count, w + len(here), tokens + count, rows + len(here)
    if step:
        yield step


class HybridRunner(DecoderRunner):
    """A hybrid decoder on one GPU; ``dtype`` torch.bfloat16, or torch.float32 for true 32-bit throughout."""

    PREFIX = "teeny_hybrid"

    def __init__(self, cfg, max_batch, max_len, max_tokens=None, max_rows=None, max_new_tokens=256, dtype=torch.bfloat16,
                 device=None):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"hybrid decoders run in bfloat16 or float32, not {dtype}")
        self.cfg, self.dtype, self.max_batch = cfg, dtype, max_batch
        self.max_tokens = max(max_batch, max_tokens if max_tokens is not None else min(max_batch * max_len, 65536))
        self.max_rows = max(max_batch, max_rows or 0)
        branches = [b for layer in cfg.layers for b in layer.branches]
        c = _Cfg(len(cfg.layers), len(branches), cfg.width, cfg.vocab, cfg.eps, cfg.embed_scale, cfg.residual_mult, int(dtype == torch.float32),
                 max_batch, max_len, self.max_tokens, self.max_rows, max_new_tokens)
        ls, bs, at = (_Layer * len(cfg.layers))(), (_Branch * len(branches))(), 0
        for i, layer in enumerate(cfg.layers):
            ls[i] = _Layer(at, len(layer.branches), layer.ff, layer.act, layer.flags)
            at += len(layer.branches)
        for i, b in enumerate(branches):
            bs[i] = _Branch(b.kind, b.heads, b.kv_heads, b.dim, b.vdim, b.rank, b.q_rank, b.window, b.rot_dims, b.flags,
                            b.score_scale, b.out_scale, b.decay_coef, b.unit_eps, b.softcap, b.rot_scale)
        nbytes = lib.teeny_hybrid_workspace_bytes(C.byref(c), ls, bs)
        if nbytes == 0:
            raise ValueError("unsupported hybrid decoder configuration for this backend")
        self.slot_bytes = lib.teeny_hybrid_slot_bytes(C.byref(c), ls, bs)
        self._init_runner(nbytes, max_len, max_new_tokens, device)
        self._h = vp()
        check(lib.teeny_hybrid_create(C.byref(c), ls, bs, C.c_void_p(self.workspace.data_ptr()), nbytes, stream(),
                                      C.byref(self._h)), "teeny_hybrid_create")
        self._free = list(range(max_batch))[::-1]
        self._rows = self._tokens = 0
        self._last_post = None  # weight of the norm behind the model's last sublayer, if it has one

    # ---- weights ----
    def _set(self, layer, branch, which, t):
        self._call("set_weight", self._h, layer, branch, which, self._upload(t))

    def load_layer(self, i, norm1, branches, norm2=None, gate=None, up=None, down=None, norm1_post=None, norm2_post=None):
        """``branches``: per branch a dict with ``inputs`` (matrices in the order of ``Branch.input_sizes``), ``out`` [width,
        output size], and the vectors (and ``low``; ``uq`` [heads * (rot_dims + dim), q_rank], ``uk``, ``uv``) its kind has; with
        IN_BIAS ``biases``, a vector or None per input."""
        layer = self.cfg.layers[i]
        if len(branches) != len(layer.branches):
            raise ValueError(f"layer {i} has {len(layer.branches)} branches, got {len(branches)}")
        for b, w in zip(layer.branches, branches):
            got = [tuple(p.shape) for p in w["inputs"]]
            want = [(n, self.cfg.width) for n in b.input_sizes()]
            if got != want or tuple(w["out"].shape) != (self.cfg.width, b.output_size()):
                raise ValueError(f"layer {i}: weight shapes {got}, {tuple(w['out'].shape)}; the configuration says {want}, "
                                 f"{(self.cfg.width, b.output_size())}")
        self._set(i, 0, W_NORM1, norm1.float())
        if layer.flags & IN_BIAS:
            bias = [torch.zeros(n, 1) if v is None else v.cpu().reshape(-1, 1) for b, w in zip(layer.branches, branches)
                    for n, v in zip(b.input_sizes(), w.get("biases") or [None] * len(w["inputs"]))]
            self._set(i, 0, W_IN_BIAS, fuse_rows(bias, self.dtype)[:, 0])
        if layer.flags & POST_NORM:
            self._set(i, 0, W_NORM1_POST, norm1_post.float())
            if layer.ff:
                self._set(i, 0, W_NORM2_POST, norm2_post.float())
            if i == len(self.cfg.layers) - 1:
                self._last_post = (norm2_post if layer.ff else norm1_post).float().to(self.device)
        self._set(i, 0, W_IN, fuse_rows([p for w in branches for p in w["inputs"]], self.dtype))
        self._set(i, 0, W_OUT, fuse_columns([w["out"] for w in branches], self.dtype))
        for j, (b, w) in enumerate(zip(layer.branches, branches)):
            for name, which in BRANCH_VECTORS.items():
                if name in w:
                    v = w[name].float().reshape(-1)
                    self._set(i, j, which, torch.nn.functional.pad(v, (0, pad_to(len(v), 8) - len(v))))
            if "low" in w:
                self._set(i, j, W_LOW, pad_columns(w["low"], 8, self.dtype))
            if b.kind == DECAY:
                self._set(i, j, BRANCH_VECTORS["decay"], torch.tensor(b.decay, dtype=torch.float64).float())
            if b.kind == LATENT:
                self._set(i, j, W_UQ, pad_columns(w["uq"], 8, self.dtype))
                for which, t in zip((W_EXPAND, W_ABSORB, W_VALUE_UP), latent_weights(b, w["uk"], w["uv"], self.dtype)):
                    self._set(i, j, which, t)
            if b.kind in (ATTENTION, LATENT) and b.rot_dims:
                self._set(i, j, BRANCH_VECTORS["inv_freq"], torch.tensor(b.frequencies(), dtype=torch.float64).float())
        if layer.ff:
            self._set(i, 0, W_NORM2, norm2.float())
            self._set(i, 0, W_GATE_UP, interleave_glu(gate, up, self.dtype))
            self._set(i, 0, W_DOWN, pad_columns(down, 64, self.dtype))

    def load_head(self, embed, final_norm, lm_head):
        self._set(0, 0, W_EMBED, embed.to(self.dtype))
        # the logits are linear in the normed rows: their scale goes with the norm's weight
        self._set(0, 0, W_FINAL_NORM, final_norm.float() * self.cfg.logit_scale)
        self._set(0, 0, W_LM_HEAD, pad_columns(lm_head, 8, self.dtype))

    # ---- sequences ----
    def open(self):
        if not self._free:
            raise RuntimeError(f"all {self.max_batch} state slots are in use")
        return Sequence(self._free.pop())

    def close(self, seq):
        """Gives the slot back; its next sequence starts at position 0, which ignores what the slot holds."""
        if seq.slot in self._free:
            raise ValueError("the sequence is closed already")
        self._free.append(seq.slot)

    def _run(self, ids, seqs, lens, rows):
        """One step of the C runner: ``ids`` device int32, entry i = the next lens[i] tokens of seqs[i]."""
        n = len(seqs)
        arr = lambda v: (i32 * max(len(v), 1))(*v)  # noqa: E731
        self._call("step", self._h, C.c_void_p(ids.data_ptr()), arr([s.slot for s in seqs]), arr([s.pos for s in seqs]), arr(lens),
                   n, arr(rows), len(rows), stream())
        self.batch = 0
        self._rows, self._tokens = len(rows), int(sum(lens))
        for s, c in zip(seqs, lens):
            s.pos += c

    def _check_ids(self, ids):
        if ids.numel() and (int(ids.min()) < 0 or int(ids.max()) >= self.cfg.vocab):
            raise ValueError("token id outside the vocabulary")
        return ids

    def step(self, entries):
        """``entries``: (sequence, token ids, wanted places among them in ascending order).  Runs the tokens from the state
        earlier steps left; returns the wanted places' logits, float32 [wanted, vocab] per entry, on the device."""
        toks = [self._check_ids(torch.as_tensor(t, dtype=torch.int32).reshape(-1)) for _, t, _ in entries]
        for s, t in zip((e[0] for e in entries), toks):
            if t.numel() == 0 or s.pos + t.numel() > self.max_len:
                raise ValueError(f"{t.numel()} tokens at position {s.pos}: the runner was created with max_len={self.max_len}")
        out = [[] for _ in entries]
        for portion in plan_steps([(t.numel(), list(w)) for t, (_, _, w) in zip(toks, entries)], self.max_tokens, self.max_rows):
            ids = torch.cat([toks[e][at:at + c] for e, at, c, _ in portion]).to(self.device)
            rows, row0 = [], 0
            for e, at, c, want in portion:
                rows += [row0 + p - at for p in want]
                row0 += c
            self._run(ids, [entries[e][0] for e, _, _, _ in portion], [c for _, _, c, _ in portion], rows)
            if rows:
                got, r = self.logits().to(torch.float32, copy=True), 0  # the next step rewrites the buffer
                for e, _, _, want in portion:
                    out[e].append(got[r:r + len(want)])
                    r += len(want)
        empty = torch.empty(0, self.cfg.vocab, device=self.device)
        return [torch.cat(o) if o else empty for o in out]

    # ---- buffers ----
    def logits(self):
        """Element type [rows, vocab]: logits of the last step's wanted rows (of every sequence after a decode step)."""
        ld = pad_to(self.cfg.vocab, 8)
        return self._view(BUF_LOGITS, (self.batch or self._rows, ld), self.dtype)[:, :self.cfg.vocab]

    def residual_stream(self):
        """float32 [tokens, width]: the residual stream after the last layer of the last step."""
        n, ld = self.batch or self._tokens, pad_to(self.cfg.width, 8)
        delta = self._view(BUF_LAST_DELTA, (n, ld), self.dtype)[:, :self.cfg.width].float()
        if self._last_post is not None:
            delta = delta * torch.rsqrt(delta.pow(2).mean(-1, keepdim=True) + self.cfg.eps) * self._last_post * self.cfg.residual_mult
        return self._view(BUF_RESIDUAL, (n, self.cfg.width), torch.float32) + delta

    # ---- generation ----
    def prefill(self, prompts, seqs):
        """Runs the prompts (int [B, S] or a list of unequal ones) into ``seqs`` and picks every first token."""
        B = len(seqs)
        if isinstance(prompts, torch.Tensor):
            rows = prompts.to(torch.int32)
            lens = [rows.shape[1]] * B
        else:
            rows = [torch.as_tensor(p, dtype=torch.int32).reshape(-1) for p in prompts]
            lens = [int(r.numel()) for r in rows]
        # the last step holds an equal share of every prompt's end, so that all first tokens are picked together
        tail = [min(n, self.max_tokens // B) for n in lens]
        head = [n - t for n, t in zip(lens, tail)]
        if any(head):
            self.step([(s, r[:h], []) for s, r, h in zip(seqs, rows, head) if h])
        if isinstance(rows, torch.Tensor):
            ids = rows[:, head[0]:].to(self.device, non_blocking=True).contiguous().view(-1)
        else:
            ids = torch.cat([r[h:] for r, h in zip(rows, head)]).to(self.device)
        ends = torch.tensor(tail).cumsum(0) - 1
        before = self.batch
        self._run(ids, seqs, tail, ends.tolist())
        self._call("begin", self._h, stream())
        self.batch = before
        self._set_batch(B)

    def _generate_group(self, prompts, max_new_tokens, use_graph):
        seqs = [self.open() for _ in range(len(prompts))]
        try:
            self.prefill(prompts, seqs)
            return self._decode_loop(max_new_tokens, use_graph)
        finally:
            for s in seqs[::-1]:
                self.close(s)

    def generate(self, prompts, max_new_tokens, use_graph=True):
        """``prompts``: int [B, S], or a list of prompts of any lengths.  Returns int32 [B, max_new_tokens] on the device.
        More prompts than state slots run in groups."""
        lens = [prompts.shape[1]] * len(prompts) if isinstance(prompts, torch.Tensor) else [len(p) for p in prompts]
        if max_new_tokens > self.max_new_tokens:
            raise ValueError("max_new_tokens exceeds the runner's history capacity")
        if not lens or min(lens) == 0 or max(lens) + max_new_tokens - 1 > self.max_len:
            raise ValueError(f"prompts of {lens} tokens + {max_new_tokens} new ones; the runner was created with max_len={self.max_len}")
        if not (isinstance(prompts, torch.Tensor) and prompts.is_cuda):  # device-resident ids are clamped by the kernel
            for p in prompts:
                self._check_ids(torch.as_tensor(p))
        room = len(self._free)
        if not room:
            raise RuntimeError(f"all {self.max_batch} state slots are in use")
        groups = [prompts[i:i + room] for i in range(0, len(lens), room)]
        if len(groups) == 1:
            return self._generate_group(prompts, max_new_tokens, use_graph)
        return torch.cat([self._generate_group(g, max_new_tokens, use_graph).clone() for g in groups])
