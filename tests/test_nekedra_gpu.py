"""Nekedra on the GPU against the plain implementation of ``plain_nekedra``.

Kernels alone (through ``Ops``), every mechanism as a one-layer model, then whole models: prompts
whole, decoded token by token, in portions down to two tokens, unequal requests in one batch on
few pages and fewer state slots than requests, long decoding through CUDA graphs, greedy
generation through ``LLM.generate`` and the trace program.  Where random weights would hide a
fault the weights are made to show it: queries are scaled up until every softmax is nearly one
key, and decays are moved close to one so that a state lost hundreds of tokens ago shows.
"""

import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import plain_nekedra as PN
import tiny_nekedra as N
from engine_helpers import Replayer, tokens_for

pytestmark = pytest.mark.gpu

# largest |engine - plain| of a row as a fraction of the largest |logit|: float32 differs from
# the float64 oracle by the order of its sums, bfloat16 by the rounding of products and
# activations.
TOL = {"float32": 5e-5, "bfloat16": 4e-2}
LOOSE_ROWS = {"float32": 0.0, "bfloat16": 0.02}


def close(got, want, dtype, what, tol=None):
    want = torch.as_tensor(np.asarray(want)).double()
    got = got.double()
    assert got.shape == want.shape, (what, got.shape, want.shape)
    scale = want.abs().max().item()
    err = (got - want).abs().max(dim=1).values / scale
    tol = tol or TOL[dtype]
    bad = int((~(err <= tol)).sum())
    assert bad <= LOOSE_ROWS[dtype] * len(err), (
        f"{what}: {bad} rows of {len(err)} differ by more than {tol:.0e} of the largest logit "
        f"(worst {err.max().item():.3e}); first wrong row {int((~(err <= tol)).nonzero()[0])}")
    assert err.max().item() < 5 * tol, f"{what}: worst row off by {err.max().item():.3e}"


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("nekedra")
    out = {}

    def sharp_and_slow(factor):
        def patch(w):
            N.sharp(factor)(w)
            N.slow_decay(w)
        return patch

    # (the wide models' sums are longer: smaller weights give scores of the same size)
    for key, raw, patch, std in (("mixed", N.N_MIXED, None, 0.15), ("plain", N.N_PLAIN, None, 0.15),
                                 ("wide", N.N_WIDE, None, 0.08),
                                 ("sharp", N.N_MIXED, sharp_and_slow(4.0), 0.15),
                                 ("sharp_wide", N.N_WIDE, sharp_and_slow(4.0), 0.08)):
        for dtype in ("float32", "bfloat16"):
            folder = tmp / f"{key}_{dtype}"
            cfg, w = N.make_nekedra(folder, raw, 11, dtype, std=std, patch=patch)
            out[(key, dtype)] = (folder, cfg, w)
    return out


# ------------------------------------------------------------------ kernels alone
@pytest.fixture(scope="module")
def rt32():
    from mini_llm_stack_b200.ops.kernels import Runtime
    return Runtime("cuda:0", torch.float32)


def fake_step(lens, starts, slots):
    """A step of ``lens[i]`` tokens from position ``starts[i]`` on for request i in ``slots[i]``."""
    from mini_llm_stack_b200.parts.base import StepContext
    i32 = dict(dtype=torch.int32, device="cuda")
    cu = np.concatenate([[0], np.cumsum(lens)])
    t = int(cu[-1])
    pos = [s + i for n, s in zip(lens, starts) for i in range(n)]
    req = [r for r, n in enumerate(lens) for _ in range(n)]
    return StepContext(
        n_tokens=t, n_requests=len(lens), token_ids=torch.zeros(t, **i32),
        positions=torch.tensor(pos, **i32), req_of_token=torch.tensor(req, **i32),
        cu_q=torch.tensor(cu.tolist(), **i32), ctx_len=torch.zeros(len(lens) + 1, **i32),
        state_slot=torch.tensor(slots, **i32), out_rows=torch.zeros(1, **i32), n_out=0,
        q_lens=list(lens), max_q_len=max(lens))


class DeltaCase:
    """Random projections of whole sequences, and what the mixer makes of them up to the gated
    heads."""

    def __init__(self, heads, kv, e, f, taps, n_tokens, seed=0, eps=1e-5):
        g = torch.Generator().manual_seed(seed)
        self.sizes, self.taps, self.eps = (heads, kv, e, f), taps, eps
        c = 2 * kv * e + heads * f
        self.cols = (4, 4 + c + heads * f + heads, 4 + c + heads * f, 4 + c)
        self.width = 4 + c + heads * f + 2 * heads + 3
        self.conv = torch.randn(c, taps, generator=g) * 0.6
        self.a_log, self.dt = torch.randn(heads, generator=g) - 2, torch.randn(heads, generator=g)
        self.norm = 1 + 0.2 * torch.randn(f, generator=g)
        self.proj = [torch.randn(n, self.width, generator=g) for n in n_tokens]
        self.want = [self._plain(p.double().numpy()) for p in self.proj]
        self.dev = {k: getattr(self, k).cuda() for k in ("conv", "dt", "norm")}
        self.dev["a_exp"] = self.a_log.exp().cuda()
        self.dev["norm_row"] = self.norm.repeat(heads).cuda()

    def _plain(self, p):
        nh, nk, e, f = self.sizes
        t, c0 = len(p), self.cols[0]
        c = 2 * nk * e + nh * f
        y = PN.silu(PN.causal_conv(p[:, c0:c0 + c], self.conv.double().numpy()))
        q = PN.unit_vector(y[:, :nk * e].reshape(t, nk, e)) * e ** -0.5
        k = PN.unit_vector(y[:, nk * e:2 * nk * e].reshape(t, nk, e))
        v = y[:, 2 * nk * e:].reshape(t, nh, f)
        g = PN.decay(p[:, self.cols[1]:self.cols[1] + nh], self.a_log.double().numpy(),
                     self.dt.double().numpy())
        b = PN.sigmoid(p[:, self.cols[2]:self.cols[2] + nh])
        o = np.stack([PN.delta_rule(q[:, h // (nh // nk)], k[:, h // (nh // nk)], v[:, h], b[:, h],
                                    g[:, h]) for h in range(nh)], axis=1)
        gate = PN.silu(p[:, self.cols[3]:self.cols[3] + nh * f]).reshape(t, nh, f)
        y = PN.unit_rms(o, self.eps) * self.norm.double().numpy() * gate
        return o.reshape(t, nh * f), y.reshape(t, nh * f)

    def new_state(self, ops, slots):
        return torch.zeros(slots, ops.delta_state_floats(*self.sizes, self.taps), device="cuda")

    def rows_of(self, portions):
        return torch.cat([self.proj[i][a:b] for i, a, b in portions]).contiguous().cuda()

    def prompt(self, ops, state, portions, slots, act):
        """Prepare, scan and finish ``portions`` [(sequence, from, to)]; (o, gated heads)."""
        step = fake_step([b - a for _, a, b in portions], [a for _, a, _ in portions], slots)
        p, (nh, nk, e, f) = self.rows_of(portions), self.sizes
        rows = torch.full((step.n_tokens, ops.delta_rows(*self.sizes)), float("nan"), device="cuda")
        ops.delta_prep(p, self.cols, self.dev["conv"], self.taps, self.dev["a_exp"], self.dev["dt"],
                       state, step, nh, nk, e, f, rows)
        o = torch.full((step.n_tokens, nh * f), float("nan"), device="cuda")
        ops.delta_scan(rows, p, self.cols[0], self.taps, state, step, nh, nk, e, f, o)
        y = torch.full((step.n_tokens, nh * f), float("nan"), dtype=act, device="cuda")
        ops.scan_finish(o, p, self.cols[3], self.dev["norm_row"], self.eps, y, nh, f)
        return o.cpu().double().numpy(), y.cpu().double().numpy()

    def single(self, ops, state, portions, slots, act, parts=None):
        step = fake_step([1] * len(portions), [a for _, a, _ in portions], slots)
        p, (nh, nk, e, f) = self.rows_of(portions), self.sizes
        if parts:
            from mini_llm_stack_b200.ops.kernels import SplitParts
            shares = [p * 0.25 for _ in range(parts - 1)]
            p = SplitParts(torch.stack([*shares, p - sum(shares)]).contiguous(), None)
        y = torch.full((len(portions), nh * f), float("nan"), dtype=act, device="cuda")
        ops.delta_step(p, self.cols, self.dev["conv"], self.taps, self.dev["a_exp"], self.dev["dt"],
                       self.dev["norm"], self.eps, state, step, nh, nk, e, f, y)
        return y.cpu().double().numpy()


DELTA_SIZES = [(4, 2, 12, 20, 3), (3, 3, 40, 8, 4), (2, 1, 64, 64, 1), (4, 2, 64, 128, 2),
               (2, 2, 100, 17, 9), (6, 1, 128, 128, 4), (1, 1, 130, 33, 5), (2, 1, 200, 136, 16),
               (2, 2, 256, 256, 4), (5, 5, 1, 1, 7), (8, 2, 32, 16, 4)]


@pytest.mark.parametrize("sizes", DELTA_SIZES)
def test_delta_kernels_over_portions_and_single_tokens(rt32, sizes):
    """Two sequences of unequal length in one batch, cut at odd places into portions (down to two
    tokens, shorter and longer than the convolution, across the prepared runs and the scan's
    buffers), then single tokens, then a portion again; slots out of order."""
    ops = rt32.ops
    ops.require_part("delta")
    nh, nk, e, f, taps = sizes
    case = DeltaCase(nh, nk, e, f, taps, (80, 41), seed=e)
    state = case.new_state(ops, 3)
    at, o, y = [0, 0], [[], []], [[], []]

    def feed(counts, single=False, parts=None):
        live = [i for i, n in enumerate(counts) if n]
        portions = [(i, at[i], at[i] + counts[i]) for i in live]
        slots = [(2, 0)[i] for i in live]
        if single:
            got = case.single(ops, state, portions, slots, torch.float32, parts)
            got_o = None
        else:
            got_o, got = case.prompt(ops, state, portions, slots, torch.float32)
        row = 0
        for i in live:
            y[i].append(got[row:row + counts[i]])
            row += counts[i]
            at[i] += counts[i]
        return got_o

    for counts in ((37, 2), (2, 17), (0, 3), (16, 0), (3, 1)):
        feed(counts)
    for k in range(8):
        feed((1, 1), single=True, parts=3 if k % 3 == 1 else None)
    feed((5, 2))
    for _ in range(8):
        feed((1, 0) if at[1] >= 41 else (1, 1), single=True)
    feed((80 - at[0], 41 - at[1]))
    assert at == [80, 41]
    for i in range(2):
        want = case.want[i][1]
        got = np.concatenate(y[i])
        # a head whose state is still nearly orthogonal to the query is a quotient of small
        # numbers: the error is measured against what the norm divides by
        rms = np.sqrt((case.want[i][0].reshape(-1, nh, f) ** 2).mean(-1) + case.eps)
        err = np.abs(got - want).reshape(-1, nh, f).max(-1) * rms
        assert np.isfinite(got).all() and err.max() < 2e-5, (i, err.max(), int(err.max(1).argmax()))


def test_delta_scan_alone_and_a_used_slot(rt32):
    """The scan's own output over a long sequence with decays near one; a slot that was used and
    cleared starts from nothing, another slot keeps what it has."""
    ops = rt32.ops
    case = DeltaCase(2, 1, 48, 24, 4, (300,), seed=3)
    case.a_log -= 6.0
    case.dev["a_exp"] = case.a_log.exp().cuda()
    case.want = [case._plain(case.proj[0].double().numpy())]
    state = case.new_state(ops, 2)
    first, _ = case.prompt(ops, state, [(0, 0, 300)], [1], torch.float32)
    scale = np.abs(case.want[0][0]).max()
    assert np.abs(first - case.want[0][0]).max() < 1e-5 * scale
    assert float(state[0].abs().max()) == 0.0
    kept = state[1].clone()
    again, _ = case.prompt(ops, state, [(0, 0, 300)], [0], torch.float32)
    assert np.array_equal(first, again) and torch.equal(state[1], kept)
    state[1].zero_()
    third, _ = case.prompt(ops, state, [(0, 0, 120), ], [1], torch.float32)
    rest, _ = case.prompt(ops, state, [(0, 120, 300)], [1], torch.float32)
    # an even cut leaves the scan's pairs of tokens as they are and changes no bit; an odd one
    # changes no more than the last bits
    assert np.array_equal(np.concatenate([third, rest]), first)
    state[1].zero_()
    odd = [case.prompt(ops, state, [(0, a, b)], [1], torch.float32)[0]
           for a, b in ((0, 121), (121, 124), (124, 300))]
    assert np.abs(np.concatenate(odd) - first).max() < 2e-6 * scale


@pytest.mark.parametrize("e", [20, 64, 90, 128])
def test_delta_scan_does_not_depend_on_the_batch(rt32, e):
    """Alone (every block of columns has an SM to itself) and beside eleven others (it has not): the
    same bits."""
    ops = rt32.ops
    case = DeltaCase(4, 2, e, 64, 3, (37,), seed=4)
    state = case.new_state(ops, 12)
    alone, _ = case.prompt(ops, state, [(0, 0, 37)], [5], torch.float32)
    kept = state[5].clone()
    state.zero_()
    many, _ = case.prompt(ops, state, [(0, 0, 37)] * 12, list(range(12)), torch.float32)
    assert all(np.array_equal(many[37 * i:37 * (i + 1)], alone) for i in range(12))
    assert torch.equal(state, kept.expand(12, -1))


def test_delta_bfloat16_outputs(rt32):
    ops = rt32.ops
    case = DeltaCase(4, 2, 64, 32, 4, (20,), seed=9)
    state = case.new_state(ops, 1)
    _, y = case.prompt(ops, state, [(0, 0, 19)], [0], torch.bfloat16)
    last = case.single(ops, state, [(0, 19, 20)], [0], torch.bfloat16)
    want = case.want[0][1]
    assert np.abs(np.concatenate([y, last]) - want).max() < 8e-3 * np.abs(want).max()


@pytest.mark.parametrize("d", [4, 40, 36, 37, 256, 1000, 2048, 4096, 5000, 8192, 9001])
@pytest.mark.parametrize("form", ["plain", "parts", "rows", "bare", "bf16"])
def test_gated_norm_kernel(rt32, d, form):
    g = torch.Generator().manual_seed(d)
    ops = rt32.ops
    t, eps = 5, 1e-3
    act = torch.bfloat16 if form == "bf16" else torch.float32
    x, y = torch.randn(t, d, generator=g), torch.randn(t, d, generator=g).to(act)
    z = torch.randn(t, d + 12, generator=g).to(act)
    bias = torch.randn(d, generator=g)
    w1 = torch.tensor([1.3]) if form != "plain" else torch.randn(d, generator=g)
    w2 = torch.tensor([0.7]) if form != "rows" else torch.randn(d, generator=g)
    zd = z.double()[:, 8:8 + d] + (0 if form == "bare" else bias.double())
    want_y = y.double() * (1 if form == "bare" else torch.sigmoid(zd))
    want_y = want_y / torch.sqrt((want_y ** 2).mean(-1, keepdim=True) + eps) * w1.double()
    want_x = x.double() + want_y
    want_h = want_x / torch.sqrt((want_x ** 2).mean(-1, keepdim=True) + eps) * w2.double()
    rows = torch.tensor([3, 0, 3], dtype=torch.int32) if form == "rows" else None
    from mini_llm_stack_b200.ops.kernels import SplitParts

    def parts(m):
        a, b = m * 0.3, m * 0.5
        return SplitParts(torch.stack([a, b, m - a - b]).contiguous().cuda(), None)
    gate = None if form == "bare" else (z.cuda(), 8)
    ydev = y.cuda()
    if form == "parts":
        ydev, gate = parts(y), parts(z[:, 8:8 + d].contiguous())
    xd = x.cuda()
    h = torch.full((3 if rows is not None else t, d), float("nan"), dtype=act, device="cuda")
    ops.add_gated_norm(xd, ydev, gate, None if form == "bare" else bias.cuda(), w1.cuda(), w2.cuda(),
                       eps, h, rows=None if rows is None else rows.cuda(), n_rows=3)
    if rows is None:
        assert (xd.cpu().double() - want_x).abs().max() < 2e-5
    else:
        assert torch.equal(xd.cpu(), x)
        want_h, want_y = want_h[rows.long()], want_y[rows.long()]
    tol = 1e-5 if act == torch.float32 else 8e-3
    assert (h.cpu().double() - want_h).abs().max() < tol * want_h.abs().max() + 1e-5
    if form in ("plain", "bare"):
        out = torch.empty(t, d, device="cuda")
        ops.add_gated_norm(None, y.cuda(), gate, None if form == "bare" else bias.cuda(), w1.cuda(),
                           None, eps, None, y_out=out)
        assert (out.cpu().double() - want_y).abs().max() < 2e-5


@pytest.mark.parametrize("per, heads, act", [(1, 24, torch.float32), (8, 3, torch.float32),
                                             (6, 5, torch.bfloat16), (128, 4, torch.bfloat16)])
def test_gate_shared_by_a_head(rt32, per, heads, act):
    g = torch.Generator().manual_seed(per)
    o = torch.randn(5, heads * per, generator=g).to(act)
    proj = torch.randn(5, heads + 9, generator=g)
    dev = o.cuda()
    rt32.ops.require_part("latent")
    rt32.ops.sigmoid_gate(dev, proj.cuda(), 8, per=per)
    want = o.double() * torch.sigmoid(proj[:, 8:8 + heads].double()).repeat_interleave(per, dim=1)
    tol = 1e-6 if act == torch.float32 else 8e-3
    assert (dev.cpu().double() - want).abs().max() < tol * want.abs().max()


def test_two_products_left_as_parts_at_once():
    """A product's parts and a gate's wait side by side; a third product under a lent name takes
    the ordinary way."""
    from mini_llm_stack_b200.ops.kernels import Runtime, SplitParts
    ops = Runtime("cuda:0", torch.bfloat16).ops
    g = torch.Generator().manual_seed(2)
    a = torch.randn(3, 2048, generator=g).bfloat16().cuda()
    ws = [(torch.randn(256, 2048, generator=g) * 0.05).bfloat16().cuda() for _ in range(3)]
    outs = [torch.empty(3, 256, device="cuda") for _ in range(3)]
    p = [ops.linear_parts(a, ws[0], outs[0]), ops.linear_parts(a, ws[1], outs[1], lend="gate"),
         ops.linear_parts(a, ws[2], outs[2])]
    assert isinstance(p[0], SplitParts) and isinstance(p[1], SplitParts) and p[2] is outs[2]
    for got, w in zip(p, ws):
        want = a.double().cpu() @ w.double().cpu().T
        got = got.float().double().cpu()
        assert (got - want).abs().max() < 1e-3 * want.abs().max()
    assert not ops._parts_busy


# ------------------------------------------------------------------ each mechanism as a model
ONE_LAYER = {
    "delta": N.one_layer(N.delta(4, 2, 20, 12, 4)),
    "delta one tap": N.one_layer(N.delta(2, 2, 32, 16, 1), 24),
    "delta 128": N.one_layer(N.delta(4, 1, 128, 128, 4), 48, width=64),
    "delta odd": N.one_layer(N.delta(3, 1, 7, 5, 6), width=34),
    "latent": N.one_layer(N.latent(4, 12, 4, 10, 20, 0.4)),
    "latent 96": N.one_layer(N.latent(2, 24, 16, 32, 80, 0.2, base=1e6), 24),
    "latent 272": N.one_layer(N.latent(3, 8, 32, 8, 240, 0.2), width=64),
    "latent 576": N.one_layer(N.latent(2, 16, 64, 24, 512, 0.15), width=64),
    "attention": N.one_layer(N.attention(6, 2, 12, 20, 0.4)),
    "attention filling": N.one_layer(N.attention(4, 4, 16, 16, 0.3, v_mix=True), 20),
    "attention 128": N.one_layer(N.attention(4, 2, 128, 96, 0.09), width=64),
    "attention mixing": N.model([N.layer(N.attention(4, 2, 20, 12, 0.3, v_mix=True)),
                                 N.layer(N.attention(2, 2, 12, 12, 0.3, v_mix=True))]),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", list(ONE_LAYER))
def test_each_mechanism(tmp_path, key, dtype):
    cfg, w = N.make_nekedra(tmp_path / "m", ONE_LAYER[key], 7, dtype)
    n = 70
    tokens = {k: tokens_for(cfg["vocab"], n, 3) for k in "abc"}
    want = PN.forward(cfg, w, tokens["a"])
    r = Replayer(tmp_path / "m", dtype, num_blocks=16)
    r.step([("a", n)], tokens, end=["a"])
    close(r.logits("a"), want, dtype, f"{key} whole")
    for s in (1, 2, 30, 3, 17, 9, 8):
        r.step([("b", s)], tokens)
    r.runner.release("b")
    close(r.logits("b"), want, dtype, f"{key} portions")
    for _ in range(n):
        r.step([("c", 1)], tokens)
    close(r.logits("c"), want, dtype, f"{key} token by token")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_residual_stream_after_every_layer(models, dtype):
    folder, cfg, w = models[("mixed", dtype)]
    from mini_llm_stack_b200.engine.batch import Entry
    from mini_llm_stack_b200.engine.runner import ModelRunner, load_model
    tokens = tokens_for(cfg["vocab"], 30, 8)
    _, want = PN.forward(cfg, w, tokens, want_layers=True)
    model = load_model(folder, dtype=dtype)
    got = []

    def listen(block):
        inner = block.forward

        def forward(stream, step, cache):
            inner(stream, step, cache)
            # settle what is pending: the next norm then finds a plain stream
            got.append((stream.x + stream.take_pending().float()).clone())
            stream.x.copy_(got[-1])
        block.forward = forward
    for b in model.blocks:
        listen(b)
    r = ModelRunner(model, num_blocks=4, max_requests=1, cuda_graphs=False)
    e = [Entry("a", tokens, [29])]
    r.reserve(e)
    r.step(e)
    assert len(got) == len(want)
    for i, (a, b) in enumerate(zip(got, want)):
        close(a.cpu(), b, dtype, f"after layer {i}")


# ------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["mixed", "plain", "wide"])
def test_whole_prompts(models, key, dtype):
    folder, cfg, w = models[(key, dtype)]
    r = Replayer(folder, dtype, num_blocks=24)
    for rid, n in (("a", 1), ("b", 2), ("c", 95), ("d", 150)):
        tokens = {rid: tokens_for(cfg["vocab"], n, n)}
        r.step([(rid, n)], tokens, end=[rid])
        close(r.logits(rid), PN.forward(cfg, w, tokens[rid]), dtype, f"{key} {n} tokens")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["mixed", "plain", "wide"])
def test_decoding_token_by_token(models, key, dtype):
    """From the very first token on: convolutions, states and pages are built by single steps."""
    folder, cfg, w = models[(key, dtype)]
    tokens = {"a": tokens_for(cfg["vocab"], 80, 4)}
    r = Replayer(folder, dtype, num_blocks=12)
    for _ in range(80):
        r.step([("a", 1)], tokens)
    close(r.logits("a"), PN.forward(cfg, w, tokens["a"]), dtype, f"{key} decoded")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(2, 2, 2, 3, 5, 7, 16, 17, 31, 33, 2, 1, 1, 40),
                                   (64, 1, 1, 1, 15, 2, 48, 28), (21, 1, 40, 17, 3, 78)])
def test_portions_of_every_size(models, sizes, dtype):
    folder, cfg, w = models[("sharp", dtype)]
    n = sum(sizes)
    tokens = {"a": tokens_for(cfg["vocab"], n, 9)}
    r = Replayer(folder, dtype, num_blocks=12)
    for s in sizes:
        r.step([("a", s)], tokens)
    if dtype == "float32":
        close(r.logits("a"), PN.forward(cfg, w, tokens["a"]), dtype, f"portions {sizes}")
    else:
        # with sharp weights a bfloat16 run is held against the engine's own whole-prompt run
        whole = Replayer(folder, dtype, num_blocks=12)
        whole.step([("a", n)], tokens)
        close(r.logits("a"), whole.logits("a").numpy(), dtype, f"portions {sizes}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["mixed", "sharp_wide"])
def test_unequal_requests_in_one_batch_on_few_pages_and_slots(models, key, dtype):
    """Five requests through three state slots and a pool that holds less than their sum:
    portions beside single tokens, requests that pause, pages and slots used again."""
    folder, cfg, w = models[(key, dtype)]
    lens = {"a": 75, "b": 33, "c": 2, "d": 58, "e": 41}
    tokens = {k: tokens_for(cfg["vocab"], n, i) for i, (k, n) in enumerate(lens.items())}
    r = Replayer(folder, dtype, num_blocks=12, max_requests=3)
    r.step([("a", 30), ("b", 2)], tokens)
    r.step([("a", 1), ("b", 17), ("c", 2)], tokens, end=["c"])
    r.step([("a", 1), ("b", 1)], tokens)
    r.step([("b", 13)], tokens, end=["b"])                     # a pauses
    r.step([("a", 40), ("d", 1), ("e", 5)], tokens)            # slots and pages of b and c again
    r.step([("e", 1), ("a", 1), ("d", 30)], tokens)
    r.step([("a", 2), ("d", 27), ("e", 35)], tokens, end=["a", "d", "e"])
    alone = Replayer(folder, dtype, num_blocks=12, max_requests=1)
    for k, n in lens.items():
        alone.step([(k, n)], tokens, end=[k])
        if dtype == "float32":
            close(r.logits(k), PN.forward(cfg, w, tokens[k]), dtype, f"{key} request {k}")
            # the batch, the cut and the pages change nothing beyond the last bits
            close(r.logits(k), alone.logits(k).numpy(), dtype, f"{key} {k} alone", tol=1e-5)
        else:
            close(r.logits(k), alone.logits(k).numpy(), dtype, f"{key} request {k}")
    assert r.runner.cache.slots.num_free == 3 and r.runner.cache.num_free_pages() == 12


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["sharp", "sharp_wide"])
def test_far_keys_and_old_states(models, key, dtype):
    """A long prompt and decoding past it with sharp softmaxes and slow decays: keys and state
    contents from hundreds of tokens back, across page borders."""
    folder, cfg, w = models[(key, dtype)]
    n = 260
    tokens = {"a": tokens_for(cfg["vocab"], n, 21)}
    r = Replayer(folder, dtype, num_blocks=20)
    r.step([("a", 200)], tokens)
    for _ in range(60):
        r.step([("a", 1)], tokens)
    if dtype == "float32":
        close(r.logits("a"), PN.forward(cfg, w, tokens["a"]), dtype, "far keys")
    else:
        whole = Replayer(folder, dtype, num_blocks=20)
        whole.step([("a", n)], tokens)
        close(r.logits("a"), whole.logits("a").numpy(), dtype, "far keys")


def test_a_single_far_key_is_found(tmp_path):
    """One token whose key stands out, hundreds of tokens back: the logits at every later place
    depend on it, in a prompt and in decoded tokens, at a page's first and last slot."""
    raw = N.model([N.layer(N.attention(2, 1, 16, 16, 1.0)),
                   N.layer(N.latent(2, 16, 4, 16, 24, 1.0))], width=32, vocab=40)

    def stand_out(w):
        N.sharp(3.0)(w)
        w["embed"][7] = 6.0 * torch.sign(w["embed"][7])
        w["embed"][8:] *= 0.2
    cfg, w = N.make_nekedra(tmp_path / "m", raw, 3, "float32", patch=stand_out)
    r = Replayer(tmp_path / "m", "float32", num_blocks=24)
    for i, place in enumerate((0, 15, 16, 31, 100)):
        other = tokens_for(30, 330, 50)
        tokens = {f"r{i}": [t + 8 for t in other]}
        without = PN.forward(cfg, w, tokens[f"r{i}"])
        tokens[f"r{i}"][place] = 7
        want = PN.forward(cfg, w, tokens[f"r{i}"])
        assert np.abs(want - without)[310:].max() > 1e-2 * np.abs(want).max()
        r.step([(f"r{i}", 300)], tokens)
        for _ in range(30):
            r.step([(f"r{i}", 1)], tokens)
        r.runner.release(f"r{i}")
        close(r.logits(f"r{i}"), want, "float32", f"far key at {place}")


def test_long_decoding_through_graphs(models):
    folder, cfg, w = models[("wide", "bfloat16")]
    lens = {"a": 150, "b": 131}
    tokens = {k: tokens_for(cfg["vocab"], n, i + 30) for i, (k, n) in enumerate(lens.items())}
    r = Replayer(folder, "bfloat16", num_blocks=24)
    r.step([("a", 20), ("b", 1)], tokens)
    for _ in range(130):
        r.step([("a", 1), ("b", 1)], tokens)
    for k in lens:
        close(r.logits(k), PN.forward(cfg, w, tokens[k]), "bfloat16", f"long decoding {k}")


@pytest.mark.parametrize("key", ["mixed", "plain"])
def test_greedy_generation_through_the_scheduler(models, key):
    from mini_llm_stack_b200.engine.llm import LLM
    folder, cfg, w = models[(key, "float32")]
    prompts = [tokens_for(cfg["vocab"], n, n + 50) for n in (3, 19, 1, 26)]
    llm = LLM.from_folder(folder, dtype="float32", num_blocks=10, block_size=16, max_batch=3)
    got = llm.generate(prompts, max_new_tokens=12)
    for p, new in zip(prompts, got):
        seq = list(p)
        logits = PN.forward(cfg, w, seq + new[:-1])
        for i, tok in enumerate(new):
            row = logits[len(p) - 1 + i]
            top = np.sort(row)[-2:]
            if top[1] - top[0] > 1e-4 * np.abs(row).max():        # not a close call
                assert tok == int(np.argmax(row)), (key, len(p), i)
    llm.engine.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_program_replays_a_folder(models, tmp_path, dtype):
    folder, cfg, w = models[("mixed", dtype)]
    a, b = tokens_for(cfg["vocab"], 50, 1), tokens_for(cfg["vocab"], 9, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[30:48], "want": []},
                                     {"id": "b", "tokens": b[:8], "want": [7]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[48:49], "want": [0]},
                                     {"id": "b", "tokens": b[8:], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[49:], "want": [0]}], "end": ["a"]}]
    root = Path(__file__).resolve().parent.parent
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(folder),
                           "--dtype", dtype, "--out", str(out), "--max-tokens", "128"],
                          input="\n".join(json.dumps(s) for s in steps) + "\n", text=True,
                          capture_output=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [ln for ln in proc.stdout.splitlines() if ln.startswith("done")] == \
        [f"done {i}" for i in range(4)]
    la, lb = PN.forward(cfg, w, a), PN.forward(cfg, w, b)
    want = {0: la[[0, 29]], 1: lb[[7]], 2: np.stack([la[48], lb[8]]), 3: la[[49]]}
    for i, rows in want.items():
        got = np.frombuffer((out / f"{i}.f32").read_bytes(), dtype="<f4").reshape(-1, cfg["vocab"])
        tol = 5e-5 if dtype == "float32" else 6e-2
        assert np.abs(got - rows).max() < tol * np.abs(rows).max(), i


def test_command_line_and_seeded_sampling(models):
    """The command line picks the model class by config.json; temperature sampling with a seed
    gives the same tokens however the requests are batched."""
    from mini_llm_stack_b200.engine.llm import LLM
    folder, cfg, w = models[("mixed", "float32")]
    root = Path(__file__).resolve().parent.parent
    p = tokens_for(cfg["vocab"], 9, 4)
    llm = LLM.from_folder(folder, dtype="float32", num_blocks=16, block_size=16, max_batch=4)
    want = llm.generate([p], max_new_tokens=6)[0]
    proc = subprocess.run(
        [sys.executable, "-m", "mini_llm_stack_b200.api", "chat", "--model", str(folder),
         "--dtype", "float32", "--token-ids", ",".join(map(str, p)), "--max-new", "6"],
        capture_output=True, text=True, cwd=root, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert proc.stdout.strip().endswith(f"-> {','.join(map(str, want))!r}")
    prompts = [tokens_for(cfg["vocab"], n, n) for n in (5, 21, 2)]
    alone = LLM.from_folder(folder, dtype="float32", num_blocks=16, block_size=16, max_batch=1)
    got = llm.generate(prompts, max_new_tokens=10, temperature=0.8, seed=5)
    one_by_one = alone.generate(prompts, max_new_tokens=10, temperature=0.8, seed=5)
    assert all(len(t) == 10 for t in got) and len(one_by_one) == 3
    llm.engine.cache.check()
