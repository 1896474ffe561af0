"""Sevazen without a GPU: configuration, tensor names, cache specs and the pages of chunks, the
rotation's scaled frequencies, the plain implementation's mechanisms on hand-made cases."""

import copy
import math

import numpy as np
import pytest

import plain_sevazen as PS
import tiny_sevazen as S
from mini_llm_stack_b200.cache.manager import CacheError, CacheManager
from mini_llm_stack_b200.config import config_from_dict
from mini_llm_stack_b200.config.model_config import ConfigError
from mini_llm_stack_b200.config.registry import build_model
from mini_llm_stack_b200.parts.attention import plan_paged_attention
from mini_llm_stack_b200.parts.base import FixedState, PagedKV, PagedWithState, StepContext
from mini_llm_stack_b200.parts.position import BandScaling, PartialRotary, YarnScaling


@pytest.mark.parametrize("raw", [S.S_MIXED, S.S_BARE, S.S_WIDE])
def test_config_round_trip(raw):
    cfg = config_from_dict(raw)
    assert cfg.architecture == "Sevazen"
    assert config_from_dict(cfg.to_dict()) == cfg
    assert config_from_dict(dict(raw, architecture="sevazen")).layers == cfg.layers


def test_layers_that_share_tensors():
    cfg = config_from_dict(S.S_MIXED)
    assert [cfg.owner(i) for i in range(7)] == [0, 1, 2, 3, 0, 1, 0]
    model = build_model(cfg)
    assert len(model.blocks) == 4
    assert [(c.layer, c.cache_slot, c.writes) for c in model.calls] == \
        [(0, 0, True), (1, 1, True), (2, 2, True), (3, 3, True), (0, 4, True), (1, 5, True), (0, 6, True)]
    assert not any(n.startswith(("l4.", "l5.", "l6.")) for n in model.tensor_specs())
    # a layer may use a later layer's tensors
    bare = build_model(config_from_dict(S.S_BARE))
    names = list(bare.tensor_specs())
    assert not any(n.startswith("l1.") for n in names) and "l3.mix.q" in names
    assert bare.calls[1].layer == bare.calls[3].layer and len(bare.cache_specs()) == 7
    chain = copy.deepcopy(S.S_MIXED)
    chain["layers"][6]["weights_of"] = 4                   # by way of layer 4, layer 0's
    assert config_from_dict(chain).owner(6) == 0


def _broken(path, value):
    raw = copy.deepcopy(S.S_MIXED)
    node = raw
    for k in path[:-1]:
        node = node[k]
    if value is KeyError:
        del node[path[-1]]
    else:
        node[path[-1]] = value
    return raw


@pytest.mark.parametrize("path, value, word", [
    (("layers", 2, "type"), "delta", "type"),
    (("layers", 2, "mixer", "kv_heads"), 3, "multiple"),
    (("layers", 2, "mixer", "conv"), 0, "conv"),
    (("layers", 3, "mixer", "conv"), 3, "does not know"),
    (("layers", 2, "mixer", "scale"), KeyError, "lacks"),
    (("layers", 2, "mixer", "diff"), 0.3, "does not know"),
    (("layers", 3, "mixer", "diff"), KeyError, "lacks"),
    (("layers", 2, "mixer", "mask"), {"size": 0}, "size"),
    (("layers", 2, "mixer", "mask"), {"size": 4, "keep_first": 1}, "does not know"),
    (("layers", 2, "mixer", "rot", "dims"), 7, "even"),
    (("layers", 2, "mixer", "rot", "dims"), 22, "at most dim"),
    (("layers", 2, "mixer", "rot", "base"), 0.0, "base"),
    (("layers", 3, "mixer", "rot", "scaling"), S.bands(2.0, 1.0, 4.0, 64), "scaling"),
    (("layers", 2, "mixer", "rot", "scaling"), S.bands(2.0, 4.0, 4.0, 64), "differ"),
    (("layers", 3, "mlp", "kind"), "gated", "kind"),
    (("layers", 3, "mlp", "router", "top"), 6, "at most"),
    (("layers", 3, "mlp", "router", "groups"), {"count": 1}, "does not know"),
    (("layers", 4, "weights_of"), 4, "weights_of"),
    (("layers", 4, "weights_of"), 7, "weights_of"),
    (("layers", 4, "weights_of"), 1, "must equal"),
    (("layers", 0, "weights_of"), 4, "leads back"),
    (("norm",), {"eps": 1e-5, "kind": "rms"}, "does not know"),
    (("embedding",), {"scale": 2.0}, "does not know"),
    (("vocab",), KeyError, "vocab"),
])
def test_config_refusals_name_the_key(path, value, word):
    with pytest.raises(ConfigError) as err:
        config_from_dict(_broken(path, value))
    assert word in str(err.value)


def test_tensor_names_and_shapes():
    specs = {n: tuple(s.shape) for n, s in
             build_model(config_from_dict(S.S_MIXED)).tensor_specs().items()}
    assert specs["embed"] == (97, 44) and "head" not in specs
    assert specs["final.norm"] == specs["final.norm.b"] == (44,)
    assert specs["l0.norm1"] == specs["l0.norm1.b"] == specs["l0.norm2.b"] == (44,)
    assert specs["l0.mix.q"] == (72, 44) and specs["l0.mix.q.b"] == (72,)
    assert specs["l0.mix.k"] == (36, 44) and specs["l0.mix.v"] == (60, 44)
    assert specs["l0.mix.k.conv"] == (36, 3) and specs["l0.mix.v.conv"] == (60, 3)
    assert specs["l0.mix.q.norm"] == specs["l0.mix.k.norm"] == (12,) and specs["l0.mix.sink"] == (6,)
    assert specs["l0.mix.o"] == (44, 120) and "l0.mix.g" not in specs
    assert specs["l0.mlp.router"] == (7, 44) and specs["l0.mlp.router.b"] == (7,)
    assert specs["l0.mlp.e6.up"] == (12, 44) and specs["l0.mlp.e6.down"] == (44, 12)
    assert "l0.mlp.e0.gate" not in specs and specs["l0.mlp.shared.up"] == (20, 44)
    assert specs["l0.mlp.shared.sg"] == (1, 44) and "l3.mlp.shared.sg" not in specs
    assert specs["l1.mix.q"] == (4 * 2 * 8, 44) and specs["l1.mix.k"] == (2 * 2 * 8, 44)
    assert specs["l1.mix.v"] == (24, 44) and specs["l1.mix.q.norm"] == (8,)
    assert specs["l1.mix.lq1"] == specs["l1.mix.lk2"] == (8,) and specs["l1.mix.g"] == (48, 44)
    assert specs["l1.mix.o"] == (44, 48) and "l1.mix.sink" not in specs and "l1.mix.q.conv" not in specs
    assert specs["l1.mlp.up"] == (28, 44) and specs["l1.mlp.down"] == (44, 28)
    assert "l2.norm2" not in specs and not any(n.startswith("l2.mlp") for n in specs)


def test_cache_specs_and_slots():
    specs = build_model(config_from_dict(S.S_MIXED)).cache_specs()
    # heads of 12 / 20 padded to 32; two rows of 72 + 36 + 60 channels
    assert specs[0] == specs[4] == specs[6] == \
        PagedWithState(PagedKV(3, 32, 19), FixedState((2 * 168,)))
    # two maps of 8 beside values of 12, padded to 16
    assert specs[1] == specs[5] == PagedKV(2, 16, chunk=24)
    assert specs[3] == PagedKV(1, 32, chunk=37)
    bare = build_model(config_from_dict(S.S_BARE)).cache_specs()
    assert bare[0] == PagedKV(1, 16) and bare[2] == PagedKV(1, 16, 1) and bare[4] == PagedKV(5, 16)
    cm = CacheManager(specs, num_blocks=12, block_size=4, max_requests=2, max_seq_len=64)
    handles = cm.handles()
    # layers with the same tensors have pages' members and tails of their own
    assert handles[0].k_pool.data_ptr() != handles[4].k_pool.data_ptr()
    assert handles[0].state.data_ptr() != handles[6].state.data_ptr()
    cm.admit("a")
    assert cm.reserve("a", 9)
    handles[4].state.fill_(7.0)
    cm.commit("a", 9)
    cm.free("a")
    cm.admit("b")                                  # a claimed slot starts from zero
    assert float(handles[4].state[cm.row("b")].abs().max()) == 0.0
    cm.check()


def test_pages_of_earlier_chunks_go_back():
    spec = PagedKV(1, 16, chunk=10)
    assert [spec.first_key(p) for p in (0, 9, 10, 19, 20)] == [0, 0, 10, 10, 20]
    assert spec.span == 10 and PagedKV(1, 16, window=7).first_key(9) == 3
    cm = CacheManager([spec, PagedKV(1, 16)], num_blocks=20, block_size=4, max_requests=2,
                      max_seq_len=80)
    cm.admit("a")
    held = []
    for n in range(1, 31):
        assert cm.reserve("a", 1)
        cm.commit("a", 1)
        pages = cm.pages_of("a", 0)
        held.append([i for i, p in enumerate(pages) if p >= 0])
        cm.check()
    # after 9 tokens the next one is the first chunk's last; after 10 the second chunk begins at
    # token 10, in page 2: pages 0 and 1 are read no more
    assert held[8] == [0, 1, 2] and held[9] == [2] and held[18] == [2, 3, 4] and held[19] == []
    assert held[20] == [5] and held[29] == [7]
    assert len([p for p in cm.pages_of("a", 1) if p >= 0]) == 8
    cm.truncate("a", 30)
    with pytest.raises(CacheError):
        cm.truncate("a", 29)                       # token 29 would read its chunk's pages again
    cm.free("a")
    assert cm.num_free_pages() == 20
    # a request fed in portions never holds more than a chunk, a portion and a page's edge
    assert cm._most_pages(cm.paged[0], 60, 8) == cm.pages_for(10 - 1 + 8) + 1
    cm.check()


def test_plan_counts_the_tiles_a_span_leaves():
    facts = {"tensor_cores": True, "small_rows": 16, "tile_rows": 64, "tc_rows": 128, "split_keys": 64,
             "split_slots": 296, "cluster_splits": 8, "cluster_slots": 296}
    none = dict.fromkeys(("token_ids", "positions", "req_of_token", "cu_q", "ctx_len", "state_slot",
                          "out_rows"))
    step = StepContext(n_tokens=2, n_requests=2, n_out=2, q_lens=[1, 1], ctx_lens=[8000, 8000],
                       max_q_len=1, max_ctx_len=8000, **none)
    far = plan_paged_attention(step, facts, 8, 2, 64)
    near = plan_paged_attention(step, facts, 8, 2, 64, span=200)
    assert far.n_split > 4 and near.n_split == 1


# ------------------------------------------------------------- the rotation's frequencies
@pytest.mark.parametrize("dims, base, args", [
    (16, 1e4, (8.0, 1.0, 4.0, 256)), (6, 300.0, (4.0, 0.5, 2.0, 64)), (2, 50.0, (3.0, 2.0, 8.0, 1000)),
    (128, 5e5, (8.0, 1.0, 4.0, 8192))])
def test_band_scaling(dims, base, args):
    factor, low, high, original = args
    got = PartialRotary(dims, base, scaling=BandScaling(factor, low, high, original))
    want, amplitude = PS.frequencies(S.rot(dims, base, S.bands(factor, low, high, original)))
    assert np.allclose(got.frequencies().numpy(), want, rtol=1e-12) and got.amplitude == amplitude == 1.0


def test_band_scaling_has_three_bands():
    plain = PS.base_frequencies(16, 1e4)
    got = [PS.banded_frequency(f, 8.0, 1.0, 4.0, 256) for f in plain]
    kinds = [g / f for g, f in zip(got, plain)]
    assert kinds[0] == 1.0 and kinds[-1] == pytest.approx(1 / 8)
    assert any(0.126 < k < 0.999 for k in kinds)
    # continuous where the bands meet
    for edge in (256 / 4.0, 256 / 1.0):
        a, b = (PS.banded_frequency(2 * math.pi / (edge * s), 8.0, 1.0, 4.0, 256) for s in (0.9999, 1.0001))
        assert a == pytest.approx(b, rel=1e-3)


@pytest.mark.parametrize("dims, base, args", [
    (8, 2e3, (8.0, 512, 16.0, 1.0)), (64, 1e4, (4.0, 4096, 32.0, 1.0)), (2, 100.0, (2.0, 64, 4.0, 1.0)),
    (20, 50.0, (16.0, 100000, 32.0, 1.0)), (12, 1e6, (0.5, 32, 1.0, 0.9))])
def test_yarn_scaling(dims, base, args):
    factor, original, fast, slow = args
    got = PartialRotary(dims, base, scaling=YarnScaling(factor, original, fast, slow))
    want, amplitude = PS.frequencies(S.rot(dims, base, S.yarn(factor, original, fast, slow)))
    assert np.allclose(got.frequencies().numpy(), want, rtol=1e-12)
    assert got.amplitude == pytest.approx(amplitude) == pytest.approx(0.1 * math.log(factor) + 1.0)


def test_yarn_keeps_fast_pairs_and_stretches_slow_ones():
    plain = PS.base_frequencies(64, 1e4)
    got = PS.yarn_frequencies(64, 1e4, 4.0, 4096, 32.0, 1.0)
    kinds = [g / f for g, f in zip(got, plain)]
    assert kinds[0] == 1.0 and kinds[-1] == pytest.approx(0.25)
    assert all(a >= b - 1e-12 for a, b in zip(kinds, kinds[1:])) and any(0.26 < k < 0.99 for k in kinds)


def test_mixers_without_an_amplitude_refuse_it():
    from mini_llm_stack_b200.parts.conv_attention import ConvKeyAttention
    pos = PartialRotary(8, 1e4, pairing="interleaved", scaling=YarnScaling(4.0, 64, 8.0, 1.0))
    with pytest.raises(ValueError, match="cosine and sine"):
        ConvKeyAttention(32, 2, 1, 16, 0.25, 1e-6, position=pos)


# ------------------------------------------------------------- the plain mechanisms
def test_window_and_chunk_edges():
    assert [PS.window_start(3)(i) for i in range(5)] == [0, 0, 0, 1, 2]
    assert [PS.chunk_start(3)(i) for i in range(7)] == [0, 0, 0, 3, 3, 3, 6]
    q, k = np.zeros((7, 1, 2)), np.zeros((7, 1, 2))
    v = np.arange(7.0).reshape(7, 1, 1)
    assert np.allclose(PS.visible_softmax(q, k, v, 1.0, PS.window_start(3))[:, 0, 0],
                       [0, 0.5, 1, 2, 3, 4, 5])
    assert np.allclose(PS.visible_softmax(q, k, v, 1.0, PS.chunk_start(3))[:, 0, 0],
                       [0, 0.5, 1, 3, 3.5, 4, 6])


def test_sink_is_not_scaled_and_counts_once():
    q, k, v = np.ones((2, 1, 2)), np.zeros((2, 1, 2)), np.full((2, 1, 3), 8.0)
    out = PS.visible_softmax(q, k, v, 5.0, lambda i: 0, sink=[math.log(3.0)])
    assert np.allclose(out[0], 2.0) and np.allclose(out[1], 8.0 * 2 / 5)


def test_convolution_meets_the_current_token_last_and_starts_from_zeros():
    x = np.array([[1.0], [10.0], [100.0]])
    y = PS.causal_conv(x, np.array([[0.5, 2.0]]))
    assert np.allclose(y[:, 0], [2.0, 20.5, 205.0])
    # the bias belongs to what is convolved: before the start there is nothing, not the bias
    h, w = np.ones((2, 1)), {"q": np.array([[2.0]]), "q.b": np.array([3.0]), "q.conv": np.array([[1.0, 1.0]])}
    assert np.allclose(PS.projected(h, w, "q", 2)[:, 0], [5.0, 10.0])
    assert np.allclose(PS.projected(h, w, "q", None)[:, 0], [5.0, 5.0])


def test_rotation_turns_halves():
    x = np.zeros((3, 5))
    x[:, 0] = 1.0
    x[:, 1] = 1.0
    x[:, 4] = 9.0
    y = PS.rotate_halves(x, S.rot(4, 100.0))
    assert np.allclose(y[2], [math.cos(2), math.cos(0.2), math.sin(2), math.sin(0.2), 9.0])
    z = PS.rotate_halves(x, S.rot(4, 100.0, S.yarn(math.e ** 10, 1e9, 32.0, 1.0)))
    assert np.allclose(z[0], [2.0, 2.0, 0.0, 0.0, 9.0])    # amplitude 2, entries past dims untouched


def test_layer_norm_and_difference():
    y = PS.layer_norm(np.array([1.0, 3.0]), np.array([2.0, 2.0]), np.array([0.5, 0.0]), 0.0)
    assert np.allclose(y, [-1.5, 2.0])
    w = {"lq1": np.array([1.0, 2.0]), "lk1": np.array([0.5, 0.0]), "lq2": np.zeros(2), "lk2": np.ones(2)}
    assert PS.lambda_of(w, 0.3) == pytest.approx(math.exp(0.5) - 1.0 + 0.3)


def test_routing_weighs_the_chosen_logits_only():
    h = np.array([[1.0]])
    w = {"router": np.array([[0.0], [1.0], [0.5]]), "router.b": np.array([2.0, 0.0, 0.0]),
         **{f"e{i}.up": np.array([[1.0]]) for i in range(3)},
         **{f"e{i}.down": np.array([[10.0 ** i]]) for i in range(3)}}
    mlp = S.moe(3, 2, 1)
    margins = []
    p = np.exp([2.0, 1.0]) / np.exp([2.0, 1.0]).sum()
    assert np.allclose(PS.routed_units(h, w, mlp, margins), p[0] + 10 * p[1])
    assert np.allclose(margins, [0.5])
    w.update({"shared.up": np.array([[2.0]]), "shared.down": np.array([[1.0]]),
              "shared.sg": np.array([[0.0]])})
    assert np.allclose(PS.routed_units(h, w, dict(mlp, shared={"ff": 1})), p[0] + 10 * p[1] + 2.0)


@pytest.fixture(scope="module")
def base(tmp_path_factory):
    cfg, w = S.make_sevazen(tmp_path_factory.mktemp("s") / "m", S.S_MIXED, 5, "float32",
                            patch=S.sharp(3.0))
    tokens = list(np.random.RandomState(1).randint(0, 97, 60))
    return cfg, w, tokens, PS.forward(cfg, w, tokens)


CHANGES = ["window+1", "window-1", "chunk+1", "chunk-1", "chunks from one", "no sink", "scaled sink",
           "reversed taps", "convolution after the norm", "bias before the start", "neighbours turn",
           "no bands", "no yarn", "no amplitude", "one map", "maps by halves", "no lambda", "no gate",
           "no head norm", "no norm bias", "norm before", "softmax over all", "no router bias",
           "no shared gate", "own tensors"]


@pytest.mark.parametrize("change", CHANGES)
def test_the_oracle_feels_every_mechanism(base, change, monkeypatch):
    """What the GPU tests compare against moves, by far more than they tolerate, when a
    mechanism is left out or read another way."""
    cfg, w, tokens, want = base
    cfg, w = copy.deepcopy(cfg), dict(w)
    layers = cfg["layers"]

    def every(kind):
        return [layer["mixer"] for layer in layers if layer["type"] == kind]

    if change[:6] in ("window", "chunk+", "chunk-"):
        kind = "attention" if change.startswith("window") else "attention_2"
        for m in every(kind):
            m["mask"]["size"] += 1 if change.endswith("+1") else -1
    elif change == "chunks from one":
        monkeypatch.setattr(PS, "chunk_start", lambda size: lambda i: max(0, (i + 1) // size * size - 1))
    elif change == "no sink":
        real = PS.visible_softmax
        monkeypatch.setattr(PS, "visible_softmax", lambda q, k, v, s, f, sink=None: real(q, k, v, s, f))
    elif change == "scaled sink":
        real = PS.visible_softmax
        monkeypatch.setattr(PS, "visible_softmax", lambda q, k, v, s, f, sink=None:
                            real(q, k, v, s, f, None if sink is None else np.asarray(sink) * s))
    elif change == "reversed taps":
        real = PS.causal_conv
        monkeypatch.setattr(PS, "causal_conv", lambda x, t: real(x, t[:, ::-1]))
    elif change == "convolution after the norm":
        def late(h, w_, m, eps):
            t = h.shape[0]

            def make(n, heads, e):
                y = (h @ w_[n].T + w_[f"{n}.b"]).reshape(t, heads, e)
                if n != "v":
                    y = PS.unit_rms(y, eps) * w_[f"{n}.norm"]
                return PS.causal_conv(y.reshape(t, -1), w_[f"{n}.conv"]).reshape(t, heads, e)
            q, k = make("q", m["heads"], m["dim"]), make("k", m["kv_heads"], m["dim"])
            v = make("v", m["kv_heads"], m["vdim"])
            o = PS.visible_softmax(PS.rotate_halves(q, m["rot"]), PS.rotate_halves(k, m["rot"]), v,
                                   m["scale"], PS.window_start(m["mask"]["size"]), sink=w_["sink"])
            return o.reshape(t, -1) @ w_["o"].T
        monkeypatch.setitem(PS.MIXERS, "attention", late)
    elif change == "bias before the start":
        def biased(h, w_, name, taps):
            y = h @ w_[name].T + w_[f"{name}.b"]
            if not taps:
                return y
            before = np.repeat(w_[f"{name}.b"][None], taps, axis=0)
            return PS.causal_conv(np.concatenate([before, y]), w_[f"{name}.conv"])[taps:]
        monkeypatch.setattr(PS, "projected", biased)
    elif change == "neighbours turn":
        def neighbours(x, rot):
            y = x.copy()
            freq, amplitude = PS.frequencies(rot)
            for p in range(x.shape[0]):
                for i, f in enumerate(freq):
                    c, s = math.cos(p * f) * amplitude, math.sin(p * f) * amplitude
                    u, v = x[p, ..., 2 * i], x[p, ..., 2 * i + 1]
                    y[p, ..., 2 * i], y[p, ..., 2 * i + 1] = u * c - v * s, v * c + u * s
            return y
        monkeypatch.setattr(PS, "rotate_halves", neighbours)
    elif change in ("no bands", "no yarn"):
        for m in every("attention" if change == "no bands" else "attention_2"):
            m["rot"].pop("scaling", None)
    elif change == "no amplitude":
        real = PS.frequencies
        monkeypatch.setattr(PS, "frequencies", lambda rot: (real(rot)[0], 1.0))
    elif change == "one map":
        monkeypatch.setattr(PS, "lambda_of", lambda w_, diff: 0.0)
    elif change == "maps by halves":
        # all heads' first maps, then all second ones
        for i in (1, 3):
            m = layers[i]["mixer"]
            for n, heads in (("q", m["heads"]), ("k", m["kv_heads"])):
                e = m["dim"]
                order = np.arange(heads * 2 * e).reshape(2, heads, e).transpose(1, 0, 2).reshape(-1)
                for name in (f"l{i}.mix.{n}", f"l{i}.mix.{n}.b"):
                    w[name] = w[name][order]
    elif change == "no lambda":
        monkeypatch.setattr(PS, "lambda_of", lambda w_, diff: diff)
    elif change == "no gate":
        for i in (1, 3):
            w[f"l{i}.mix.g"] = np.zeros_like(w[f"l{i}.mix.g"])
    elif change == "no head norm":
        for n in list(w):
            if n.endswith(("q.norm", "k.norm")):
                w[n] = np.full_like(w[n], w[n].mean())
    elif change == "no norm bias":
        for n in list(w):
            if n.endswith(("norm1.b", "norm2.b")):
                w[n] = np.zeros_like(w[n])
    elif change == "norm before":
        real = PS.window_attention

        def normed(h, w_, m, eps):
            return real(PS.layer_norm(h, 1.0, 0.0, eps), w_, m, eps)
        monkeypatch.setitem(PS.MIXERS, "attention", normed)
    elif change == "softmax over all":
        def over_all(h, w_, mlp, margins=None):
            z = h @ w_["router"].T + w_["router.b"]
            p = np.exp(z - z.max(1, keepdims=True))
            p /= p.sum(1, keepdims=True)
            y = np.zeros_like(h)
            for t in range(len(h)):
                for e in np.argsort(-z[t], kind="stable")[:mlp["router"]["top"]]:
                    y[t] += p[t, e] * PS.dense_unit(h[t], {"up": w_[f"e{e}.up"], "down": w_[f"e{e}.down"]})
            if mlp.get("shared") is not None:
                y = y + PS.dense_unit(h, {"up": w_["shared.up"], "down": w_["shared.down"]}) \
                    * PS.sigmoid(h @ w_["shared.sg"].T)
            return y
        monkeypatch.setattr(PS, "routed_units", over_all)
    elif change == "no router bias":
        for n in list(w):
            if n.endswith("router.b"):
                w[n] = np.zeros_like(w[n])
    elif change == "no shared gate":
        w["l0.mlp.shared.sg"] = np.zeros_like(w["l0.mlp.shared.sg"])
    elif change == "own tensors":
        layers[4] = dict(layers[2])
        layers[4]["weights_of"] = 2
    got = PS.forward(cfg, w, tokens)
    moved = np.abs(got - want).max(axis=1) / np.abs(want).max()
    assert moved.max() > 3e-3, (change, moved.max())
    if change == "window+1":
        assert moved[:19].max() < 1e-12        # rows inside the smallest window see the same keys
    if change == "chunk+1":
        assert moved[:24].max() < 1e-12
