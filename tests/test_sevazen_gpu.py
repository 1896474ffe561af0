"""Sevazen on the GPU against the plain implementation of ``plain_sevazen``.

Kernels alone (through ``Ops``), every mechanism as a one-layer model, then whole models: prompts
whole, decoded token by token, in portions down to two tokens, unequal requests in one batch on
few pages and fewer state slots than requests, the edges of windows and chunks, long decoding
through CUDA graphs, greedy generation through ``LLM.generate`` and the trace program.  Where
random weights would hide a fault the weights are made to show it: the query norms' weights are
scaled up until every softmax is nearly one key, and single keys are made to stand out.
"""

import json
import math
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import plain_sevazen as PS
import tiny_sevazen as S
from engine_helpers import Replayer, tokens_for

pytestmark = pytest.mark.gpu

# largest |engine - plain| of a row as a fraction of the largest |logit|: float32 differs from
# the float64 oracle by the order of its sums, bfloat16 by the rounding of products and
# activations.  A router's close call could fall the other way in a bfloat16 run, so the models
# of the bfloat16 runs have routers whose choices rest on their biases (``decisive_routers``);
# the float32 runs keep routers that choose by the token.
TOL = {"float32": 5e-5, "bfloat16": 4e-2}
LOOSE_ROWS = {"float32": 0.0, "bfloat16": 0.02}
DTYPES = [torch.float32, torch.bfloat16]


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


def make(folder, raw, seed, dtype, patch=None, **kw):
    def both(w):
        if patch:
            patch(w)
        if dtype == "bfloat16":
            S.decisive_routers(w)
    return S.make_sevazen(folder, raw, seed, dtype, patch=both, **kw)


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("sevazen")
    out = {}
    # (the wide models' sums are longer: smaller weights give values of the same size)
    for key, raw, patch, std in (("mixed", S.S_MIXED, None, 0.15), ("bare", S.S_BARE, None, 0.15),
                                 ("wide", S.S_WIDE, None, 0.08),
                                 ("sharp", S.S_MIXED, S.sharp(4.0), 0.15),
                                 ("sharp_wide", S.S_WIDE, S.sharp(3.0), 0.08)):
        for dtype in ("float32", "bfloat16"):
            folder = tmp / f"{key}_{dtype}"
            cfg, w = make(folder, raw, 11, dtype, patch=patch, std=std)
            out[(key, dtype)] = (folder, cfg, w)
    return out


# ------------------------------------------------------------------ kernels alone
@pytest.fixture(scope="module")
def rts():
    from mini_llm_stack_b200.ops.kernels import Runtime
    return {d: Runtime("cuda:0", d) for d in DTYPES}


def fake_step(lens, starts, slots, cache_slots=None, block_size=4):
    """A step of ``lens[i]`` tokens from position ``starts[i]`` on for request i in state slot
    ``slots[i]``, tokens stored at ``cache_slots``."""
    from mini_llm_stack_b200.parts.base import GroupView, StepContext
    i32 = dict(dtype=torch.int32, device="cuda")
    cu = np.concatenate([[0], np.cumsum(lens)])
    t = int(cu[-1])
    pos = [s + i for n, s in zip(lens, starts) for i in range(n)]
    req = [r for r, n in enumerate(lens) for _ in range(n)]
    groups = {}
    if cache_slots is not None:
        groups[0] = GroupView(torch.zeros((len(lens), 8), **i32), torch.tensor(cache_slots, **i32),
                              block_size, 8)
    return StepContext(
        n_tokens=t, n_requests=len(lens), token_ids=torch.zeros(t, **i32),
        positions=torch.tensor(pos, **i32), req_of_token=torch.tensor(req, **i32),
        cu_q=torch.tensor(cu.tolist(), **i32), ctx_len=torch.zeros(len(lens) + 1, **i32),
        state_slot=torch.tensor(slots, **i32), out_rows=torch.zeros(1, **i32), n_out=0,
        groups=groups, q_lens=list(lens), max_q_len=max(lens))


# heads, kv heads, maps, e, f, hd, taps, rotated entries; the last ones take the kernel with its
# heads in shared memory (more than four taps, heads beyond a warp's registers)
PREP_SIZES = [(6, 3, 1, 12, 20, 32, 3, 8), (4, 2, 2, 8, 12, 16, 0, 6), (3, 1, 2, 10, 24, 32, 0, 10),
              (4, 2, 1, 64, 64, 64, 4, 32), (2, 1, 1, 128, 96, 128, 2, 128), (5, 5, 2, 7, 9, 16, 0, 0),
              (6, 3, 2, 32, 64, 64, 0, 16), (12, 1, 2, 48, 128, 128, 0, 48), (3, 1, 1, 16, 16, 16, 1, 0),
              (2, 2, 1, 20, 8, 32, 4, 4), (2, 1, 1, 36, 260, 272, 4, 36), (2, 2, 1, 5, 34, 48, 9, 4),
              (2, 1, 1, 64, 32, 64, 5, 64), (2, 1, 2, 132, 300, 304, 0, 120), (2, 2, 1, 40, 66, 80, 12, 6)]


@pytest.mark.parametrize("act", DTYPES)
@pytest.mark.parametrize("sizes", PREP_SIZES)
def test_head_preparation_over_portions_and_single_tokens(rts, sizes, act):
    """Biases, convolution with its carried tail, norms per map, rotation with an amplitude, maps side
    by side, zero padding, cleared page tails: two sequences of unequal length in one batch, cut at
    odd places into portions (down to two tokens, shorter and longer than the convolution), then
    single tokens, then a portion again; state slots out of order."""
    from mini_llm_stack_b200.parts.base import CacheHandle
    ops = rts[act].ops
    nh, nkv, maps, e, f, hd, taps, dims = sizes
    ops.require_part("headprep")
    ops.require_part("shortconv")
    g = torch.Generator().manual_seed(hd + taps)
    cq, ck, cv = nh * maps * e, nkv * maps * e, nkv * f
    c, col, bs, amp, eps = cq + ck + cv, 4, 4, 1.25, 1e-5
    width = col + c + (3 if e % 2 else 4)
    seqs = [torch.randn(n, width, generator=g) for n in (64, 33)]
    bias = torch.randn(c, generator=g)
    conv = torch.randn(c, taps, generator=g) if taps else None
    wq, wk = 1 + 0.3 * torch.randn(e, generator=g), 1 + 0.3 * torch.randn(e, generator=g)
    rotation = S.rot(dims, 50.0) if dims else None
    freq = PS.base_frequencies(dims, 50.0) if dims else None

    def plain(p):
        t = len(p)
        y = p[:, col:col + c].double().numpy() + bias.double().numpy()
        if taps:
            y = PS.causal_conv(y, conv.double().numpy())
        q = PS.unit_rms(y[:, :cq].reshape(t, nh, maps, e), eps) * wq.double().numpy()
        k = PS.unit_rms(y[:, cq:cq + ck].reshape(t, nkv, maps, e), eps) * wk.double().numpy()
        out = []
        for x in (q, k):
            r = PS.rotate_halves(x, rotation)
            if dims:
                r[..., :dims] *= amp
            out.append(r)
        return out[0], out[1], y[:, cq + ck:].reshape(t, nkv, f)
    want = [plain(p) for p in seqs]
    pages = 40
    pool = torch.full((2, nkv, pages, bs, hd), float("nan"), dtype=act, device="cuda")
    cache = CacheHandle(kind="paged", group=0, k_pool=pool[0], v_pool=pool[1])
    tail = torch.zeros(3, max(0, taps - 1) * c, device="cuda")
    dev = {"bias": bias.cuda(), "conv": conv.t().contiguous().cuda() if taps else None,
           "norms": (wq.cuda(), wk.cuda()),
           "freq": torch.tensor(freq, dtype=torch.float64, device="cuda") if dims else None}
    base = (0, 20 * bs)                       # the sequences' first cache slots
    at = [0, 0]
    tol = 2e-5 if act == torch.float32 else 1e-2

    def feed(counts):
        live = [i for i, n in enumerate(counts) if n]
        lens, starts = [counts[i] for i in live], [at[i] for i in live]
        slots = [base[i] + at[i] + j for i in live for j in range(counts[i])]
        step = fake_step(lens, starts, [(2, 0)[i] for i in live], slots, bs)
        proj = torch.cat([seqs[i][at[i]:at[i] + counts[i]] for i in live]).contiguous().cuda()
        q_row = torch.full((step.n_tokens, (nh * maps + 2 * nkv) * hd), float("nan"), dtype=act,
                           device="cuda")
        single = step.max_q_len == 1
        ops.head_conv_rope_store(proj, col, dev["bias"], dev["conv"], taps, tail, dev["norms"], eps,
                                 dev["freq"], dims, amp, q_row, cache, step, nh, nkv, e, f, hd, maps=maps,
                                 move_tail=single)
        if taps > 1 and not single:
            ops.tail_update(proj, col, c, dev["bias"], tail, taps - 1, step)
        row, q_row = 0, q_row.cpu().double().numpy()
        kv = pool.cpu().double().numpy().reshape(2, nkv, pages * bs, hd)
        for i in live:
            for j in range(counts[i]):
                p = at[i] + j
                got = q_row[row, :nh * maps * hd].reshape(nh, maps, hd)
                expect = np.zeros_like(got)
                for m in range(maps):
                    expect[:, m, m * e:(m + 1) * e] = want[i][0][p][:, m]
                assert np.isfinite(got).all()
                assert np.abs(got - expect).max() < tol * np.abs(expect).max(), ("q", i, p)
                expect = np.zeros((2, nkv, hd))
                expect[0, :, :maps * e] = want[i][1][p].reshape(nkv, maps * e)
                expect[1, :, :f] = want[i][2][p]
                got = kv[:, :, base[i] + p]
                assert np.abs(got - expect).max() < tol * np.abs(expect).max(), ("kv", i, p)
                row += 1
            at[i] += counts[i]
            # the rest of the page the sequence ends in reads as zeros
            end = base[i] + at[i]
            rest = kv[:, :, end:(end + bs - 1) // bs * bs]
            assert rest.size == 0 or np.abs(rest).max() == 0.0
    for counts in ((17, 2), (2, 9), (0, 3), (16, 0), (3, 1)):
        feed(counts)
    for _ in range(6):
        feed((1, 1))
    feed((5, 2))
    feed((1, 1))
    feed((64 - at[0], 33 - at[1]))
    ops.check_status()


def test_head_preparation_of_many_tokens_gives_the_bits_of_few(rts):
    from mini_llm_stack_b200.parts.base import CacheHandle
    ops = rts[torch.float32].ops
    g = torch.Generator().manual_seed(1)
    nh, nkv, e, f, hd, taps, t = 8, 2, 32, 32, 32, 4, 1200
    c = (nh + nkv) * e + nkv * f
    proj = torch.randn(t, c, generator=g).cuda()
    conv, freq = torch.randn(taps, c, generator=g).cuda(), torch.tensor(
        PS.base_frequencies(32, 1e4), dtype=torch.float64, device="cuda")
    tail = torch.randn(1, (taps - 1) * c, generator=g).cuda()

    def run(rows, start, slots):
        pool = torch.zeros(2, nkv, 1, 2048, hd, device="cuda")
        out = torch.zeros(rows.shape[0], (nh + 2 * nkv) * hd, device="cuda")
        step = fake_step([rows.shape[0]], [start], [0], slots, 2048)
        ops.head_conv_rope_store(rows.contiguous(), 0, None, conv, taps, tail, None, 0.0, freq, 32, 1.0,
                                 out, CacheHandle(kind="paged", group=0, k_pool=pool[0], v_pool=pool[1]),
                                 step, nh, nkv, e, f, hd)
        return out[:, :nh * hd], pool
    many, pool = run(proj, 5, list(range(t)))
    few, _ = run(proj[:3], 5, [0, 1, 2])
    assert torch.equal(many[:3], few) and float(pool[0, :, 0, t:].abs().max()) == 0.0


@pytest.mark.parametrize("d", [4, 40, 36, 37, 256, 1000, 2048, 4096, 5000, 8192, 9001])
@pytest.mark.parametrize("form", ["plain", "parts", "rows", "bare", "bf16", "final", "stream"])
def test_norm_behind_a_sublayer(rts, d, form):
    from mini_llm_stack_b200.ops.kernels import SplitParts
    g = torch.Generator().manual_seed(d)
    ops = rts[torch.float32].ops
    ops.require_part("layernorm")
    t, eps = (700 if form == "plain" and d <= 4096 else 5), 1e-3
    act = torch.bfloat16 if form == "bf16" else torch.float32
    x, y = torch.randn(t, d, generator=g) + 3.0, (torch.randn(t, d, generator=g) - 2.0).to(act)
    bias, w1, b1, w2, b2 = (torch.randn(d, generator=g) for _ in range(5))

    def norm(v, w, b):
        m = v.mean(-1, keepdim=True)
        return (v - m) / torch.sqrt(((v - m) ** 2).mean(-1, keepdim=True) + eps) * w.double() + b.double()
    has_bias, has_norm = form in ("parts", "final"), form in ("final", "rows")
    want_y = norm(y.double() + (bias.double() if has_bias else 0.0), w1, b1)
    want_x = x.double() + (0.0 if form == "stream" else want_y)
    want_h = norm(want_x, w2, b2) if has_norm else want_x
    rows = torch.tensor([3, 0, 3], dtype=torch.int32) if form == "rows" else None
    xd, yd = x.cuda(), y.cuda()
    if form == "parts":
        a, b = y * 0.3, y * 0.5
        yd = SplitParts(torch.stack([a, b, y - a - b]).contiguous().cuda(), None)
    h = torch.full((3 if rows is not None else t, d), float("nan"), dtype=act, device="cuda")
    ops.add_post_layernorm(xd, None if form == "stream" else yd,
                           None if form == "stream" else (w1.cuda(), b1.cuda()), eps, h,
                           bias=bias.cuda() if has_bias else None,
                           norm=(w2.cuda(), b2.cuda()) if has_norm else None,
                           rows=None if rows is None else rows.cuda(), n_rows=3)
    if rows is None:
        assert (xd.cpu().double() - want_x).abs().max() < 2e-5
    else:
        assert torch.equal(xd.cpu(), x)
        want_h = want_h[rows.long()]
    tol = 1e-5 if act == torch.float32 else 8e-3
    assert (h.cpu().double() - want_h).abs().max() < tol * want_h.abs().max() + 1e-5
    if form == "bare":
        out = torch.empty(t, d, device="cuda")
        ops.add_post_layernorm(None, y.cuda(), (w1.cuda(), b1.cuda()), eps, None, y_out=out)
        assert (out.cpu().double() - want_y).abs().max() < 2e-5


@pytest.mark.parametrize("act", DTYPES)
@pytest.mark.parametrize("heads, f, hd, gated", [(3, 12, 16, True), (5, 9, 16, True), (4, 128, 128, True),
                                                 (2, 64, 64, False), (1, 300, 304, True), (7, 1, 16, True)])
def test_difference_of_two_maps(rts, heads, f, hd, gated, act):
    g = torch.Generator().manual_seed(f)
    ops = rts[act].ops
    ops.require_part("headprep")
    t, lam, mul, eps = 6, 0.37, 0.6, 1e-4
    o = torch.randn(t, 2 * heads * hd, generator=g).to(act)
    z = torch.randn(t, heads * f + 8, generator=g)
    out = torch.full((t, heads * f), float("nan"), dtype=act, device="cuda")
    ops.head_difference(o.cuda(), hd, lam, mul, eps, z.cuda() if gated else None, 4, out, heads, f)
    a = o.double().numpy().reshape(t, heads, 2, hd)[..., :f]
    want = PS.unit_rms(a[:, :, 0] - lam * a[:, :, 1], eps).reshape(t, -1) * mul
    if gated:
        want = want * PS.sigmoid(z.double().numpy()[:, 4:4 + heads * f])
    tol = 1e-5 if act == torch.float32 else 8e-3
    assert np.abs(out.cpu().double().numpy() - want).max() < tol * np.abs(want).max()


@pytest.mark.parametrize("experts, top", [(1, 1), (7, 3), (16, 4), (64, 64), (40, 2)])
@pytest.mark.parametrize("biased", [True, False])
def test_routing_by_logits(rts, experts, top, biased):
    """Choice and weights against the plain rule, with ties, with logits far beyond what an exponential
    holds, and with a column behind the router's."""
    rt = rts[torch.float32]
    ops = rt.ops
    ops.require_part("experts")
    g = torch.Generator().manual_seed(experts)
    t = 33
    z = torch.randn(t, experts + 1, generator=g)
    z[1] = 0.0                                        # all equal: the lowest numbers win
    z[2] *= 300.0
    z[3] = z[3] * 300.0 - 2000.0
    b = torch.randn(experts, generator=g) if biased else None
    n = t * top
    i32 = dict(dtype=torch.int32, device="cuda")
    tiles = ops.expert_max_tiles(n, experts)
    work = {"idx": torch.zeros(n, **i32), "weight": torch.zeros(n, device="cuda"),
            "order": torch.zeros(n, **i32), "offsets": torch.zeros(experts + 1, **i32),
            "cursor": torch.zeros(experts, **i32), "tile_expert": torch.zeros(tiles, **i32),
            "tile_row0": torch.zeros(tiles, **i32), "max_tiles": tiles}
    ops.route(z.cuda(), top, False, work, correction=b.cuda() if biased else None, n_outputs=experts,
              by_logit=True)
    s = (z[:, :experts] + (b if biased else 0.0)).float()
    idx, weight = work["idx"].cpu().view(t, top), work["weight"].cpu().view(t, top)
    for i in range(t):
        order = sorted(range(experts), key=lambda e: (-float(s[i, e]), e))[:top]
        assert idx[i].tolist() == order, i
        p = torch.softmax(s[i, order].double(), 0)
        assert (weight[i].double() - p).abs().max() < 1e-5, i


@pytest.mark.parametrize("act, d, f, experts, top, t", [
    (torch.float32, 44, 12, 7, 3, 9), (torch.bfloat16, 64, 40, 5, 2, 30), (torch.bfloat16, 128, 96, 4, 2, 400),
    (torch.bfloat16, 38, 10, 3, 3, 8), (torch.float32, 64, 33, 1, 1, 5)])
def test_ungated_experts(rts, act, d, f, experts, top, t):
    rt = rts[act]
    from mini_llm_stack_b200.parts.feedforward import RoutedExperts, SquaredReluFeedForward
    part = RoutedExperts(d, experts, top, f, shared=SquaredReluFeedForward(d, 16), weigh="output",
                         score="logit", router_bias=True, shared_gate=True, unit="relu_squared")
    g = torch.Generator().manual_seed(d)
    w = {n: (torch.randn(s.shape, generator=g) * (0.2 if s.kind == "matrix" else 1.0)).to(act)
         for n, s in part.tensor_specs().items()}
    w["router.b"] = torch.arange(experts).float().to(act) * 3.0      # clear choices
    w["router"] *= 0.1
    h = torch.randn(t, d, generator=g).to(act)
    part.bind({n: v.cuda() for n, v in w.items()}, rt)
    got = part.forward(h.cuda(), None).cpu().double().numpy()
    want = PS.routed_units(h.double().numpy(), {n: v.double().numpy() for n, v in w.items()},
                           S.moe(experts, top, f, 16))
    tol = 1e-5 if act == torch.float32 else 2e-2
    assert np.abs(got - want).max() < tol * np.abs(want).max()


class SpanAttention:
    """Requests with given contexts and portions over pages the cache manager hands out; a window or
    chunks."""

    def __init__(self, rt, heads, kv, hd, block, ctxs, q_lens, chunk=None, window=None, sink=False,
                 seed=0):
        from mini_llm_stack_b200.cache.manager import CacheManager
        from mini_llm_stack_b200.parts.base import PagedKV
        self.rt, self.heads, self.kv, self.hd, self.block = rt, heads, kv, hd, block
        self.ctxs, self.q_lens, self.chunk, self.window = ctxs, q_lens, chunk, window
        g = torch.Generator().manual_seed(seed)
        act = rt.act_dtype
        self.spec = PagedKV(kv, hd, window, chunk=chunk)
        self.cache = CacheManager([self.spec], sum(-(-c // block) for c in ctxs) + 3, block,
                                  len(ctxs) + 1, max(ctxs) + 8, device="cuda", kv_dtype=act)
        self.cache.paged[0].kv.fill_(3.0)            # what an earlier owner left
        self.k = [torch.randn(kv, c, hd, generator=g).to(act) for c in ctxs]
        self.v = [torch.randn(kv, c, hd, generator=g).to(act) for c in ctxs]
        self.q = [torch.randn(heads, n, hd, generator=g).to(act) for n in q_lens]
        self.sink = torch.randn(heads, generator=g) if sink else None

    def run(self):
        from mini_llm_stack_b200.engine.batch import BatchBuilder, Entry
        from mini_llm_stack_b200.parts.attention import plan_paged_attention
        rt, cache, bs = self.rt, self.cache, self.block
        ops, handle, entries = rt.ops, cache.handles()[0], []
        for i, (c, n) in enumerate(zip(self.ctxs, self.q_lens)):
            cache.admit(i)
            assert cache.reserve(i, c - n)
            cache.commit(i, c - n)                   # pages of what is out of sight go back
            assert cache.reserve(i, n)
            entries.append(Entry(i, [0] * n, []))
        for i, c in enumerate(self.ctxs):
            for b, pg in enumerate(cache.pages_of(i)):
                if pg >= 0:
                    n = min(bs, c - b * bs)
                    handle.k_pool[:, pg, :n] = self.k[i][:, b * bs:b * bs + n].cuda()
                    handle.v_pool[:, pg, :n] = self.v[i][:, b * bs:b * bs + n].cuda()
        step = BatchBuilder(cache, "cuda", 10, 1 << 20).build(entries)
        t = step.n_tokens
        qkv = torch.zeros(t, (self.heads + 2 * self.kv) * self.hd, dtype=rt.act_dtype, device="cuda")
        qkv[:, :self.heads * self.hd] = torch.cat([q.transpose(0, 1).reshape(q.shape[1], -1)
                                                   for q in self.q]).cuda()
        out = torch.full((t, self.heads * self.hd), float("nan"), dtype=rt.act_dtype, device="cuda")
        if ops.attention_tensor_cores(self.hd):
            ops.require_attention(self.hd)
        plan = plan_paged_attention(step, ops.attention_facts(self.hd), self.heads, self.kv, self.hd,
                                    span=self.spec.span, share_groups=True)
        assert plan is None or plan.share == (1 if self.heads // self.kv <= 16 else 2)
        ops.paged_attention(qkv, out, handle, step, self.heads, self.kv, self.hd, self.hd ** -0.5,
                            self.window or 0, plan=plan, chunk=self.chunk or 0,
                            sink=self.sink.cuda() if self.sink is not None else None)
        ops.check_status()
        return out.float().cpu()

    def want(self):
        rows = []
        for q, k, v in zip(self.q, self.k, self.v):
            n, c = q.shape[1], k.shape[1]
            kk, vv = (x.float().repeat_interleave(self.heads // self.kv, 0) for x in (k, v))
            s = torch.einsum("hqe,hke->hqk", q.float(), kk) * self.hd ** -0.5
            for i in range(n):
                p = c - n + i
                s[:, i, p + 1:] = -math.inf
                s[:, i, :self.spec.first_key(p)] = -math.inf
            if self.sink is not None:
                s = torch.cat([s, self.sink[:, None, None].expand(-1, n, 1)], 2)
            a = torch.softmax(s.double(), 2)[:, :, :c].float()
            rows.append((a @ vv).transpose(0, 1).reshape(n, -1))
        return torch.cat(rows)

    def check(self, what=""):
        got, want = self.run(), self.want()
        assert bool(torch.isfinite(got).all()), what
        tol = 5e-6 if self.rt.act_dtype == torch.float32 else 1.2e-2
        scale = want.abs().max(dim=1).values.clamp(min=1.0)
        err = (got - want).abs().max(dim=1).values / scale
        assert bool((err <= tol).all()), (what, float(err.max()), int(err.argmax()))
        return got


@pytest.mark.parametrize("impl", ["auto", "mma", "no_tma", "simt"])
@pytest.mark.parametrize("heads, kv, hd, block, chunk", [
    (8, 2, 64, 16, 64), (8, 2, 128, 16, 77), (4, 2, 64, 16, 300), (24, 1, 128, 16, 100), (6, 3, 32, 16, 24),
    (4, 4, 48, 8, 1), (8, 1, 64, 8, 8), (4, 2, 16, 5, 13), (2, 1, 128, 64, 512), (2, 2, 256, 16, 40)])
def test_chunked_attention_of_every_kernel(rts, impl, heads, kv, hd, block, chunk):
    """Whole prompts, portions that begin and end inside, at the edge and behind the edge of chunks,
    single tokens that are a chunk's last, first and second; pages of earlier chunks given back; the
    window beside the chunk's size shows that the two are told apart."""
    rt = rts[torch.bfloat16]
    c = chunk
    ctxs = [7, 3 * c + 200, c, c + 1, 2 * c, 2 * c + 1, 2 * c + 2, 333, 4 * c + 5, 700]
    q_lens = [7, 150, 1, 1, 1, 1, 2, 333, c + 3 if c < 200 else 3, 2]
    rt.ops.attention_impl = impl
    try:
        SpanAttention(rt, heads, kv, hd, block, ctxs, q_lens, chunk=chunk, seed=hd).check(impl)
    finally:
        rt.ops.attention_impl = "auto"


@pytest.mark.parametrize("rows", [128, 256])
@pytest.mark.parametrize("hd", [64, 128])
@pytest.mark.parametrize("chunk", [90, 128, 600])
def test_chunked_prompts_in_both_row_arrangements(rts, rows, hd, chunk):
    rt = rts[torch.bfloat16]
    rt.ops.set_attention_rows(hd, rows)
    try:
        SpanAttention(rt, 8, 2, hd, 16, [333, 45, 700, 64, 1300, 130], [70, 45, 300, 64, 515, 33],
                      chunk=chunk, seed=rows).check()
    finally:
        rt.ops.set_attention_rows(hd, 0)


@pytest.mark.parametrize("chunk, ctxs, q_lens", [(64, [64, 65, 128, 1], [1, 1, 2, 1]),
                                                 (37, [300, 111, 38], [300, 40, 1]), (1, [9, 50], [9, 1])])
def test_chunked_attention_in_float32(rts, chunk, ctxs, q_lens):
    SpanAttention(rts[torch.float32], 4, 2, 48, 16, ctxs, q_lens, chunk=chunk, seed=chunk).check()


@pytest.mark.parametrize("splits", [1, 2, 3, 8, 12])
@pytest.mark.parametrize("span", [dict(chunk=700), dict(chunk=2000), dict(window=700)])
def test_chunks_cut_into_forced_splits(rts, monkeypatch, splits, span):
    monkeypatch.setenv("MLS_B200_SPLITS", str(splits))
    for hd, heads, kv, sink in ((64, 8, 2, True), (128, 32, 8, False), (32, 6, 3, True),
                                (128, 64, 2, True), (64, 24, 1, False), (48, 40, 2, True)):
        SpanAttention(rts[torch.bfloat16], heads, kv, hd, 16, [3000, 70, 1025, 1, 1399, 2001],
                      [1, 1, 1, 1, 2, 1], seed=31, sink=sink, **span).check((hd, splits))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("span, size, ctx, q_len", [
    ("chunk", 24, 49, 1), ("chunk", 24, 48, 1), ("chunk", 100, 101, 40), ("chunk", 100, 250, 130),
    ("chunk", 64, 129, 2), ("window", 72, 200, 1), ("window", 72, 300, 150), ("window", 5, 40, 7)])
def test_keys_just_inside_and_outside(rts, dtype, span, size, ctx, q_len):
    """A key with a huge score and a huge value just outside the last query's window or chunk must not
    count; the same key just inside must."""
    for hd, heads, kv in ((32, 4, 2), (64, 8, 2), (128, 4, 1)):
        case = SpanAttention(rts[dtype], heads, kv, hd, 16, [ctx], [q_len], seed=5, **{span: size})
        first = case.spec.first_key(ctx - 1)
        q, k, v = case.q[0], case.k[0], case.v[0]
        k[:, first - 1] = q[0, -1] * 3
        v[:, first - 1] = 1000.0
        got = case.check("outside")
        assert got[-1].abs().max().item() < 100
        case = SpanAttention(rts[dtype], heads, kv, hd, 16, [ctx], [q_len], seed=5, **{span: size})
        q, k, v = case.q[0], case.k[0], case.v[0]
        k[:, first] = q[0, -1] * 3
        v[:, first] = 50.0
        got = case.check("inside")
        assert got[-1, :hd].max().item() > 40


# ------------------------------------------------------------------ each mechanism as a model
BANDS, YARN = S.bands(4.0, 1.0, 4.0, 40), S.yarn(4.0, 60, 8.0, 1.0)
ONE_LAYER = {
    "window": S.one_layer(S.window(6, 2, 12, 20, 0.4, 19, S.rot(8, 100.0, BANDS), 4)),
    "window only": S.one_layer(S.window(4, 2, 16, 16, 0.3, 24)),
    "no window, one tap": S.one_layer(S.window(2, 2, 8, 24, 0.4, None, S.rot(8, 50.0), 1), width=36),
    "window 64": S.one_layer(S.window(4, 2, 64, 48, 0.12, 33, S.rot(64, 1e3, BANDS), 4), width=64),
    "window 128": S.one_layer(S.window(4, 1, 128, 128, 0.09, 70, S.rot(32, 1e3, BANDS), 2), width=64),
    "window 304": S.one_layer(S.window(2, 1, 300, 260, 0.06, 20, S.rot(20, 1e3, BANDS), 3), width=64),
    "many taps": S.one_layer(S.window(3, 3, 10, 14, 0.3, 40, S.rot(4, 20.0, BANDS), 11)),
    "pair": S.one_layer(S.pair(4, 2, 8, 12, 0.4, 0.3, 24, S.rot(6, 100.0, YARN))),
    "pair without chunks": S.one_layer(S.pair(3, 3, 9, 10, 0.4, 0.6, None, S.rot(8, 30.0, YARN))),
    "pair 64": S.one_layer(S.pair(4, 2, 32, 64, 0.2, 0.4, 40, S.rot(32, 1e3, YARN)), width=64),
    "pair 128, wide group": S.one_layer(S.pair(20, 1, 40, 128, 0.2, 0.2, 33, S.rot(16, 1e3, YARN)), width=64),
    "pair of one token": S.one_layer(S.pair(2, 1, 16, 16, 0.3, 0.5, 1, S.rot(16, 1e3))),
    "routed": S.one_layer(S.window(2, 1, 8, 8, 0.3, 16), S.moe(9, 4, 12, 20)),
    "routed, nothing shared": S.one_layer(S.window(2, 1, 8, 8, 0.3, 16), S.moe(6, 2, 10)),
    "dense": S.one_layer(S.window(2, 1, 8, 8, 0.3, 16), S.dense(52)),
    "twice": S.model([S.layer(S.window(4, 2, 12, 12, 0.4, 12, S.rot(8, 30.0), 4), S.dense(20))] * 1
                     + [dict(S.layer(S.window(4, 2, 12, 12, 0.4, 12, S.rot(8, 30.0), 4), S.dense(20)),
                             weights_of=0)]),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", list(ONE_LAYER))
def test_each_mechanism(tmp_path, key, dtype):
    cfg, w = make(tmp_path / "m", ONE_LAYER[key], 7, dtype)
    n = 76
    tokens = {k: tokens_for(cfg["vocab"], n, 3) for k in "abc"}
    want = PS.forward(cfg, w, tokens["a"])
    r = Replayer(tmp_path / "m", dtype, num_blocks=16)
    r.step([("a", n)], tokens, end=["a"])
    close(r.logits("a"), want, dtype, f"{key} whole")
    for s in (1, 2, 30, 3, 17, 9, 14):
        r.step([("b", s)], tokens)
    r.runner.release("b")
    close(r.logits("b"), want, dtype, f"{key} portions")
    for _ in range(n):
        r.step([("c", 1)], tokens)
    close(r.logits("c"), want, dtype, f"{key} token by token")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["mixed", "bare"])
def test_residual_stream_after_every_layer(models, key, dtype):
    folder, cfg, w = models[(key, dtype)]
    from mini_llm_stack_b200.engine.batch import Entry
    from mini_llm_stack_b200.engine.runner import ModelRunner, load_model
    tokens = tokens_for(cfg["vocab"], 50, 8)
    _, want = PS.forward(cfg, w, tokens, want_layers=True)
    model = load_model(folder, dtype=dtype)
    got = []

    def listen(block):
        inner = block.forward

        def forward(stream, step, cache):
            inner(stream, step, cache)
            # settle what is pending: the next read then finds a plain stream
            got.append((stream.x + stream.take_pending().float()).clone())
            stream.x.copy_(got[-1])
        block.forward = forward
    for b in model.blocks:
        listen(b)
    r = ModelRunner(model, num_blocks=4, max_requests=1, cuda_graphs=False)
    e = [Entry("a", tokens, [49])]
    r.reserve(e)
    r.step(e)
    assert len(got) == len(want) == 7
    for i, (a, b) in enumerate(zip(got, want)):
        close(a.cpu(), b, dtype, f"after layer {i}")


# ------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["mixed", "bare", "wide"])
def test_whole_prompts(models, key, dtype):
    folder, cfg, w = models[(key, dtype)]
    r = Replayer(folder, dtype, num_blocks=24)
    for rid, n in (("a", 1), ("b", 2), ("c", 95), ("d", 170)):
        tokens = {rid: tokens_for(cfg["vocab"], n, n)}
        r.step([(rid, n)], tokens, end=[rid])
        close(r.logits(rid), PS.forward(cfg, w, tokens[rid]), dtype, f"{key} {n} tokens")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["mixed", "bare", "wide"])
def test_decoding_token_by_token(models, key, dtype):
    """From the very first token on: tails and pages are built by single steps."""
    folder, cfg, w = models[(key, dtype)]
    tokens = {"a": tokens_for(cfg["vocab"], 110, 4)}
    r = Replayer(folder, dtype, num_blocks=12)
    for _ in range(110):
        r.step([("a", 1)], tokens)
    close(r.logits("a"), PS.forward(cfg, w, tokens["a"]), dtype, f"{key} decoded")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["sharp", "sharp_wide"])
@pytest.mark.parametrize("sizes", [(2, 2, 2, 3, 5, 7, 16, 17, 31, 33, 2, 1, 1, 40),
                                   (64, 1, 1, 1, 15, 2, 48, 28), (21, 1, 40, 17, 3, 78), (2,) * 40])
def test_portions_of_every_size(models, key, sizes, dtype):
    folder, cfg, w = models[(key, dtype)]
    n = sum(sizes)
    tokens = {"a": tokens_for(cfg["vocab"], n, 9)}
    r = Replayer(folder, dtype, num_blocks=12)
    for s in sizes:
        r.step([("a", s)], tokens)
    if dtype == "float32":
        close(r.logits("a"), PS.forward(cfg, w, tokens["a"]), dtype, f"portions {sizes}")
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
            close(r.logits(k), PS.forward(cfg, w, tokens[k]), dtype, f"{key} request {k}")
            # the batch, the cut and the pages change nothing beyond the last bits
            close(r.logits(k), alone.logits(k).numpy(), dtype, f"{key} {k} alone", tol=1e-5)
        else:
            close(r.logits(k), alone.logits(k).numpy(), dtype, f"{key} request {k}")
    assert r.runner.cache.slots.num_free == 3 and r.runner.cache.num_free_pages() == 12


def test_a_pool_full_of_nan_does_not_reach_a_new_request(models):
    for key in ("mixed", "wide"):
        folder, cfg, w = models[(key, "bfloat16")]
        r = Replayer(folder, "bfloat16", num_blocks=12)
        for g in r.runner.cache.paged:
            g.kv.fill_(float("nan"))
        for g in r.runner.cache.fixed:
            g.state.fill_(float("nan"))
        tokens = {"a": tokens_for(cfg["vocab"], 90, 2)}
        for s in (37, 1, 2, 49, 1):
            r.step([("a", s)], tokens)
        close(r.logits("a"), PS.forward(cfg, w, tokens["a"]), "bfloat16", key)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["sharp", "sharp_wide"])
def test_far_keys_and_decoding_past_windows_and_chunks(models, key, dtype):
    """A long prompt and decoding past it with sharp softmaxes: windows and chunks pass over decoded
    tokens, their pages go back and are used again."""
    folder, cfg, w = models[(key, dtype)]
    n = 330
    tokens = {"a": tokens_for(cfg["vocab"], n, 21)}
    r = Replayer(folder, dtype, num_blocks=24)
    r.step([("a", 210)], tokens)
    for _ in range(120):
        r.step([("a", 1)], tokens)
    if dtype == "float32":
        close(r.logits("a"), PS.forward(cfg, w, tokens["a"]), dtype, "far keys")
    else:
        whole = Replayer(folder, dtype, num_blocks=24)
        whole.step([("a", n)], tokens)
        close(r.logits("a"), whole.logits("a").numpy(), dtype, "far keys")


def test_a_single_far_key_is_found(tmp_path):
    """One token whose keys stand out, hundreds of tokens back, in layers without limits: the logits
    at every later place depend on it, in a prompt and in decoded tokens, at a page's first and
    last slot."""
    raw = S.model([S.layer(S.window(2, 1, 16, 16, 1.0)), S.layer(S.pair(2, 1, 8, 16, 1.0, 0.3))],
                  width=32, vocab=40)

    def stand_out(w):
        S.sharp(6.0)(w)
        w["embed"][7] = 6.0 * torch.sign(w["embed"][7])
    cfg, w = make(tmp_path / "m", raw, 3, "float32", patch=stand_out)
    r = Replayer(tmp_path / "m", "float32", num_blocks=24)
    for i, place in enumerate((0, 15, 16, 31, 100)):
        tokens = {f"r{i}": [t + 8 for t in tokens_for(30, 330, 50)]}
        without = PS.forward(cfg, w, tokens[f"r{i}"])
        tokens[f"r{i}"][place] = 7
        want = PS.forward(cfg, w, tokens[f"r{i}"])
        assert np.abs(want - without)[310:].max() > 1e-3 * np.abs(want).max()
        r.step([(f"r{i}", 300)], tokens)
        for _ in range(30):
            r.step([(f"r{i}", 1)], tokens)
        r.runner.release(f"r{i}")
        close(r.logits(f"r{i}"), want, "float32", f"far key at {place}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mixer, first", [
    (S.window(2, 1, 16, 16, 0.1, 23), lambda p: max(0, p - 22)),
    (S.pair(2, 1, 16, 32, 0.1, 0.3, 23), lambda p: p // 23 * 23)])
def test_the_edges_of_windows_and_chunks(tmp_path, mixer, first, dtype):
    """One token that stands out, one layer whose softmaxes are flat: a later position's logits move
    exactly if it lies in that position's window or chunk, in a prompt and decoded one by one."""
    raw = S.model([S.layer(mixer)], width=32, vocab=40)

    def stand_out(w):
        w["embed"][7] = 4.0 * torch.sign(w["embed"][7])
    cfg, w = make(tmp_path / "m", raw, 3, dtype, patch=stand_out)
    r = Replayer(tmp_path / "m", dtype, num_blocks=24)
    n = 120
    other = [t + 8 for t in tokens_for(30, n, 50)]
    for place in (22, 23, 45, 46, 60):
        marked = list(other)
        marked[place] = 7
        for how in ("prompt", "decoded"):
            rows = {}
            for name, seq in (("plain", other), ("marked", marked)):
                rid = f"{place}{how}{name}"
                tokens = {rid: seq}
                if how == "prompt":
                    r.step([(rid, n)], tokens)
                else:
                    r.step([(rid, place + 1)], tokens)
                    for _ in range(n - place - 1):
                        r.step([(rid, 1)], tokens)
                r.runner.release(rid)
                rows[name] = r.logits(rid)
            moved = (rows["marked"] - rows["plain"]).abs().max(dim=1).values
            for p in range(place + 1, n):
                sees = first(p) <= place
                assert bool(moved[p] > 1e-3) == sees, (place, how, p, float(moved[p]))


def test_long_decoding_through_graphs(models):
    for key in ("wide", "mixed"):
        folder, cfg, w = models[(key, "bfloat16")]
        lens = {"a": 150, "b": 131}
        tokens = {k: tokens_for(cfg["vocab"], n, i + 30) for i, (k, n) in enumerate(lens.items())}
        r = Replayer(folder, "bfloat16", num_blocks=24)
        r.step([("a", 20), ("b", 1)], tokens)
        for _ in range(130):
            r.step([("a", 1), ("b", 1)], tokens)
        for k in lens:
            close(r.logits(k), PS.forward(cfg, w, tokens[k]), "bfloat16", f"long decoding {key} {k}")


def test_sequences_longer_than_the_pool_and_than_the_tables_sent(tmp_path):
    """Layers that all see a window or a chunk give their pages back, so a sequence may outgrow the
    pool; the block tables that a step sends grow with it (and captured steps with them)."""
    raw = S.model([S.layer(S.window(2, 1, 16, 16, 0.5, 20, S.rot(8, 100.0), 3)),
                   S.layer(S.pair(2, 1, 8, 16, 0.5, 0.3, 24))], width=32, vocab=40)
    make(tmp_path / "m", raw, 3, "float32")
    n = 300
    tokens = {"a": tokens_for(40, n, 1)}
    want = None
    for width, blocks in ((2048, 24), (2, 6)):
        r = Replayer(tmp_path / "m", "float32", num_blocks=blocks)
        assert r.runner.max_seq_len == 1 << 20
        r.runner.builder.width = width
        for _ in range(4):
            r.step([("a", 20)], tokens)
        for _ in range(n - 80):
            r.step([("a", 1)], tokens)
        if want is not None:
            assert torch.equal(r.logits("a"), want)
            assert r.runner.builder.width == 32                # 19 pages
        want = r.logits("a")


@pytest.mark.parametrize("key", ["mixed", "bare"])
def test_greedy_generation_through_the_scheduler(models, key):
    from mini_llm_stack_b200.engine.llm import LLM
    folder, cfg, w = models[(key, "float32")]
    prompts = [tokens_for(cfg["vocab"], n, n + 50) for n in (3, 19, 1, 26)]
    llm = LLM.from_folder(folder, dtype="float32", num_blocks=10, block_size=16, max_batch=3)
    got = llm.generate(prompts, max_new_tokens=12)
    for p, new in zip(prompts, got):
        seq = list(p)
        logits = PS.forward(cfg, w, seq + new[:-1])
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
    la, lb = PS.forward(cfg, w, a), PS.forward(cfg, w, b)
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
