"""Nekedra without a GPU: configuration, tensor names, cache specs, and the plain
implementation's mechanisms on hand-made cases."""

import copy
import math

import numpy as np
import pytest

import plain_nekedra as PN
import tiny_nekedra as N
from mini_llm_stack_b200.cache.manager import CacheManager
from mini_llm_stack_b200.config import config_from_dict
from mini_llm_stack_b200.config.model_config import ConfigError
from mini_llm_stack_b200.config.registry import build_model
from mini_llm_stack_b200.parts.base import FixedState, PagedKV


@pytest.mark.parametrize("raw", [N.N_MIXED, N.N_PLAIN, N.N_WIDE])
def test_config_round_trip(raw):
    cfg = config_from_dict(raw)
    assert cfg.architecture == "Nekedra"
    assert config_from_dict(cfg.to_dict()) == cfg
    assert config_from_dict(dict(raw, architecture="nekedra")).layers == cfg.layers


def test_mixing_layers():
    assert config_from_dict(N.N_MIXED).mixing_layers() == [1, 5, 6]
    assert config_from_dict(N.N_PLAIN).mixing_layers() == []
    blocks = build_model(config_from_dict(N.N_MIXED)).blocks
    assert [b.mixer.fills_first for b in (blocks[1], blocks[3], blocks[5], blocks[6])] == \
        [True, False, False, False]
    assert blocks[3].mixer.first_values is None
    assert blocks[1].mixer.first_values is blocks[6].mixer.first_values


def _broken(path, value):
    raw = copy.deepcopy(N.N_MIXED)
    node = raw
    for k in path[:-1]:
        node = node[k]
    if value is KeyError:
        del node[path[-1]]
    else:
        node[path[-1]] = value
    return raw


@pytest.mark.parametrize("path, value, word", [
    (("layers", 0, "type"), "conv", "type"),
    (("layers", 0, "mixer", "kv_heads"), 3, "multiple"),
    (("layers", 0, "mixer", "conv"), 0, "conv"),
    (("layers", 0, "mixer", "scale"), 1.0, "does not know"),
    (("layers", 1, "mixer", "scale"), KeyError, "lacks"),
    (("layers", 1, "mixer", "mask"), {"size": 3}, "does not know"),
    (("layers", 1, "mixer", "v_mix"), 3, "v_mix"),
    (("layers", 5, "mixer", "vdim"), 24, "same kv_heads and vdim"),
    (("layers", 2, "mixer", "rot", "dims"), 4, "rot_dim"),
    (("layers", 2, "mixer", "rot", "base"), 0.0, "base"),
    (("layers", 2, "mixer", "kv_rank"), -1, "kv_rank"),
    (("layers", 0, "mlp", "kind"), "moe", "dense"),
    (("layers", 0, "mlp", "ff"), 0, "ff"),
    (("norm",), {"eps": 1e-5, "kind": "layer"}, "does not know"),
    (("embedding",), {"scale": 2.0}, "does not know"),
    (("vocab",), KeyError, "vocab"),
])
def test_config_refusals_name_the_key(path, value, word):
    with pytest.raises(ConfigError) as err:
        config_from_dict(_broken(path, value))
    assert word in str(err.value)


def test_tensor_names_and_shapes():
    specs = {n: tuple(s.shape) for n, s in
             build_model(config_from_dict(N.N_MIXED)).tensor_specs().items()}
    assert specs["embed"] == (97, 40) and specs["head"] == (97, 40) and specs["final.norm"] == ()
    assert specs["l0.norm1"] == specs["l0.norm1b"] == specs["l0.norm2b"] == ()
    assert specs["l0.rg1"] == specs["l0.rg2"] == (40, 40) and specs["l0.rg2.b"] == (40,)
    assert specs["l0.mix.q"] == (2 * 12, 40) and specs["l0.mix.v"] == (4 * 20, 40)
    assert specs["l0.mix.k.conv"] == (2 * 12, 3) and specs["l0.mix.v.conv"] == (4 * 20, 3)
    assert specs["l0.mix.a"] == specs["l0.mix.b"] == (4, 40)
    assert specs["l0.mix.A_log"] == specs["l0.mix.dt_bias"] == (4,)
    assert specs["l0.mix.norm"] == (20,) and specs["l0.mix.g"] == (80, 40)
    assert specs["l0.mix.o"] == (40, 80)
    assert specs["l1.mix.q.b"] == (48,) and specs["l1.mix.v.b"] == (40,)
    assert specs["l1.mix.sink"] == (4,) and specs["l1.mix.vmix"] == () == specs["l6.mix.vmix"]
    assert "l3.mix.vmix" not in specs and specs["l3.mix.sink"] == (3,)
    assert "l3.norm2" not in specs and "l3.rg2" not in specs and "l3.rg1.b" in specs
    assert specs["l2.mix.q"] == (3 * 16, 40) and specs["l2.mix.dkv"] == (24, 40)
    assert specs["l2.mix.dkv.norm"] == (18,) and specs["l2.mix.g"] == (3, 40)
    assert specs["l2.mix.uk"] == (30, 18) and specs["l2.mix.uv"] == (42, 18)
    assert "l2.mix.sink" not in specs


def test_cache_specs_and_slots():
    model = build_model(config_from_dict(N.N_MIXED))
    specs = model.cache_specs()
    # 4 heads of 12 x 20 (padded to 32 x 32) and three rows of 2 * 24 + 80 channels
    assert specs[0] == FixedState((4 * 32 * 32 + 3 * 128,))
    assert specs[4] == FixedState((3 * 16 * 64 + 4 * 264,))
    assert specs[1] == PagedKV(2, 32, None) and specs[3] == PagedKV(3, 16, None)
    assert specs[2] == PagedKV(1, 32, None, shared_kv=True)
    cm = CacheManager(specs, num_blocks=8, block_size=4, max_requests=2, max_seq_len=64)
    handles = cm.handles()
    assert handles[0].state.shape == (2, 4 * 32 * 32 + 3 * 128)
    cm.admit("a")
    assert cm.reserve("a", 9)
    handles[0].state.fill_(7.0)
    cm.commit("a", 9)
    cm.free("a")
    cm.admit("b")                                  # a claimed slot starts from zero
    assert float(handles[0].state[cm.row("b")].abs().max()) == 0.0
    cm.check()


# ------------------------------------------------------------- the plain mechanisms
def test_delta_rule_replaces_what_the_key_holds():
    k = np.array([[1.0, 0.0], [1.0, 0.0], [0.0, 1.0]])
    v = np.array([[3.0], [5.0], [2.0]])
    one = np.ones(3)
    # full steps without decay: a key's second value takes the first one's place
    out = PN.delta_rule(k, k, v, one, one)
    assert np.allclose(out[:, 0], [3.0, 5.0, 2.0])
    # half a step goes half the way, after the decay
    out = PN.delta_rule(k[:2], k[:2], v[:2], np.array([1.0, 0.5]), np.array([1.0, 0.5]))
    assert np.allclose(out[1, 0], 1.5 + 0.5 * (5.0 - 1.5))


def test_convolution_meets_the_current_token_last():
    x = np.array([[1.0], [10.0], [100.0]])
    y = PN.causal_conv(x, np.array([[0.5, 2.0]]))
    assert np.allclose(y[:, 0], [2.0, 20.5, 205.0])
    assert np.allclose(PN.causal_conv(x, np.array([[3.0]])), 3.0 * x)


def test_decay_and_unit_vectors():
    assert PN.decay(np.array(0.0), 0.0, 0.0) == pytest.approx(math.exp(-math.log(2.0)))
    assert PN.decay(np.array(2.0), math.log(3.0), -1.0) == pytest.approx(
        math.exp(-3.0 * math.log(1.0 + math.e)))
    u = PN.unit_vector(np.array([3.0, 4.0]))
    assert np.allclose(u, [0.6, 0.8]) and np.allclose(PN.unit_vector(np.zeros(2)), 0.0)


def test_sink_is_not_scaled():
    q, k, v = np.ones((1, 1, 2)), np.zeros((1, 1, 2)), np.full((1, 1, 3), 8.0)
    assert np.allclose(PN.causal_softmax(q, k, v, 5.0, sink=[math.log(3.0)]), 2.0)
    assert np.allclose(PN.causal_softmax(q, k, v, 5.0), 8.0)


def test_rotation_turns_neighbours():
    x = np.zeros((3, 5))
    x[:, 0] = 1.0
    x[:, 2] = 1.0
    x[:, 4] = 9.0
    y = PN.rotate_pairs(x, 4, 100.0)
    assert np.allclose(y[2], [math.cos(2), math.sin(2), math.cos(0.2), math.sin(0.2), 9.0])


@pytest.fixture(scope="module")
def base(tmp_path_factory):
    cfg, w = N.make_nekedra(tmp_path_factory.mktemp("n") / "m", N.N_MIXED, 5, "float32",
                            patch=N.sharp(4.0))
    tokens = list(np.random.RandomState(1).randint(0, 97, 60))
    return cfg, w, tokens, PN.forward(cfg, w, tokens)


@pytest.mark.parametrize("change", [
    "no sink", "scaled sink", "no mixing", "mix from the layer before", "half rotation",
    "rotated from one", "late convolution", "no decay", "no forgetting", "read before write",
    "no unit vectors", "no head gate", "no residual gate", "key heads by turns"])
def test_the_oracle_feels_every_mechanism(base, change, monkeypatch):
    """What the GPU tests compare against moves, by far more than they tolerate, when a
    mechanism is left out or read another way."""
    cfg, w, tokens, want = base
    cfg, w = copy.deepcopy(cfg), dict(w)
    if change == "no sink":
        real = PN.causal_softmax
        monkeypatch.setattr(PN, "causal_softmax", lambda q, k, v, s, sink=None: real(q, k, v, s))
    elif change == "scaled sink":
        real = PN.causal_softmax
        monkeypatch.setattr(PN, "causal_softmax", lambda q, k, v, s, sink=None:
                            real(q, k, v, s, None if sink is None else np.asarray(sink) * s))
    elif change == "no mixing":
        for i in (5, 6):
            w[f"l{i}.mix.vmix"] = np.array(0.0)
    elif change == "mix from the layer before":
        class Last(list):
            def append(self, v):
                self[:] = [v]
        real = PN.attention_mixer

        def mixer(h, ww, m, first):
            out = real(h, ww, m, first)
            if m.get("v_mix") and first:
                t = h.shape[0]
                first[0] = (h @ ww["v"].T + ww["v.b"]).reshape(t, m["kv_heads"], m["vdim"])
            return out
        monkeypatch.setattr(PN, "attention_mixer", mixer)
    elif change == "half rotation":
        def half(x, dims, base_):
            y = x.copy()
            for p in range(x.shape[0]):
                for i in range(dims // 2):
                    a = p * base_ ** (-2.0 * i / dims)
                    u, v = x[p, ..., i], x[p, ..., i + dims // 2]
                    y[p, ..., i] = u * math.cos(a) - v * math.sin(a)
                    y[p, ..., i + dims // 2] = v * math.cos(a) + u * math.sin(a)
            return y
        monkeypatch.setattr(PN, "rotate_pairs", half)
    elif change == "rotated from one":
        # positions from one move q and k alike: only a query that misses the shift shows
        real = PN.rotate_pairs
        monkeypatch.setattr(PN, "rotate_pairs", lambda x, d, b: real(
            np.concatenate([x[:1], x]), d, b)[1:] if x.ndim == 3 else real(x, d, b))
    elif change == "late convolution":
        real = PN.causal_conv
        monkeypatch.setattr(PN, "causal_conv", lambda x, t: real(x, t[:, ::-1]))
    elif change == "no decay":
        monkeypatch.setattr(PN, "decay", lambda a, al, dt: np.ones_like(a))
    elif change == "no forgetting":
        def keep(q, k, v, beta, g):
            s, out = np.zeros((q.shape[1], v.shape[1])), np.zeros_like(v)
            for i in range(len(q)):
                s = g[i] * s + np.outer(k[i], beta[i] * v[i])
                out[i] = s.T @ q[i]
            return out
        monkeypatch.setattr(PN, "delta_rule", keep)
    elif change == "read before write":
        def early(q, k, v, beta, g):
            s, out = np.zeros((q.shape[1], v.shape[1])), np.zeros_like(v)
            for i in range(len(q)):
                out[i] = s.T @ q[i]
                s = g[i] * s
                s = s + np.outer(k[i], beta[i] * (v[i] - s.T @ k[i]))
            return out
        monkeypatch.setattr(PN, "delta_rule", early)
    elif change == "no unit vectors":
        monkeypatch.setattr(PN, "unit_vector", lambda x: x)
    elif change == "no head gate":
        w["l2.mix.g"] = np.zeros_like(w["l2.mix.g"])
        w["l2.mix.o"] = w["l2.mix.o"] * 2.0
    elif change == "no residual gate":
        monkeypatch.setattr(PN, "residual_gate", lambda y, h, ww, b: y)
    elif change == "key heads by turns":
        w["l0.mix.v"] = w["l0.mix.v"].reshape(4, 20, 40)[[0, 2, 1, 3]].reshape(80, 40)
    got = PN.forward(cfg, w, tokens)
    moved = np.abs(got - want).max(axis=1) / np.abs(want).max()
    assert moved.max() > 5e-3, change
