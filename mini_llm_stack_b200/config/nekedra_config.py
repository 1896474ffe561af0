"""Typed configuration of the Nekedra decoder, read from its config.json.

config.json: ``architecture``, ``vocab``, ``width``, ``norm.eps`` and ``layers``, a list in which
every entry names its mixer (``type``: ``delta``, ``latent_attention`` or ``attention``), the
mixer's sizes and constants (``mixer``) and its feed-forward (``mlp``: ``kind`` ``dense`` with its
width ``ff``, or null for none).

* ``delta``: ``heads`` (value heads), ``kv_heads`` (key heads), ``dim`` (queries and keys), ``vdim``
  (values) and ``conv`` (taps of the short convolutions).
* ``latent_attention``: ``heads``, ``dim`` and ``rot_dim`` (plain and rotated entries of a query
  head), ``vdim``, ``kv_rank`` (the latent), ``scale`` and ``rot`` (``base``, ``dims`` = ``rot_dim``).
* ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale`` and an optional ``v_mix`` (the
  values are mixed with those of the first layer that says so).

Every size and constant of a model comes from there.  Positions are not bounded by a table, so
a sequence is as long as the engine lets it be (``max_seq_len``, an engine-side bound that
config.json may carry).
"""

from __future__ import annotations

from dataclasses import dataclass

from .model_config import ConfigError, canonical_dtype_name

DEFAULT_MAX_SEQ_LEN = 1 << 20
TYPES = ("delta", "latent_attention", "attention")


def _need(cond, msg):
    if not cond:
        raise ConfigError(msg)


def _positive_int(v, what):
    _need(isinstance(v, int) and not isinstance(v, bool) and v > 0,
          f"{what} must be a positive integer, got {v!r}")
    return v


def _positive(v, what):
    _need(isinstance(v, (int, float)) and not isinstance(v, bool) and v > 0,
          f"{what} must be a positive number, got {v!r}")
    return float(v)


def _keys(d, want: set, what: str, optional: set = frozenset()):
    _need(isinstance(d, dict), f"{what} must be an object, got {d!r}")
    missing, unknown = want - set(d), set(d) - want - optional
    _need(not missing, f"{what} lacks {sorted(missing)}")
    _need(not unknown, f"{what} has keys this architecture does not know: {sorted(unknown)}")


def _sizes(m, names, what: str) -> None:
    for k in names:
        _positive_int(m[k], f"{what}.{k}")


def _check_groups(m, what: str) -> None:
    _need(m["heads"] % m["kv_heads"] == 0,
          f"{what}.heads ({m['heads']}) must be a multiple of kv_heads ({m['kv_heads']})")


def _check_delta(m, what: str) -> None:
    names = ("conv", "dim", "heads", "kv_heads", "vdim")
    _keys(m, set(names), what)
    _sizes(m, names, what)
    _check_groups(m, what)


def _check_latent(m, what: str) -> None:
    names = ("dim", "heads", "kv_rank", "rot_dim", "vdim")
    _keys(m, {*names, "rot", "scale"}, what)
    _sizes(m, names, what)
    _positive(m["scale"], f"{what}.scale")
    _keys(m["rot"], {"base", "dims"}, f"{what}.rot")
    _positive(m["rot"]["base"], f"{what}.rot.base")
    dims = _positive_int(m["rot"]["dims"], f"{what}.rot.dims")
    _need(dims % 2 == 0 and dims == m["rot_dim"],
          f"{what}.rot.dims ({dims}) must be even and equal rot_dim ({m['rot_dim']})")


def _check_attention(m, what: str) -> None:
    names = ("dim", "heads", "kv_heads", "vdim")
    _keys(m, {*names, "scale"}, what, optional={"v_mix"})
    _sizes(m, names, what)
    _check_groups(m, what)
    _positive(m["scale"], f"{what}.scale")
    _need(m.get("v_mix") in (None, False, True), f"{what}.v_mix must be true or false")


@dataclass(frozen=True)
class NekedraConfig:
    architecture: str = "Nekedra"
    vocab: int = 256
    width: int = 64
    layers: tuple = ()
    norm_eps: float = 1e-6
    max_seq_len: int = DEFAULT_MAX_SEQ_LEN
    dtype: str = "bfloat16"

    # what the framework reads
    @property
    def vocab_size(self) -> int:
        return self.vocab

    def __post_init__(self):
        _positive_int(self.vocab, "vocab")
        _positive_int(self.width, "width")
        _positive_int(self.max_seq_len, "max_seq_len")
        _need(self.norm_eps > 0, "norm.eps must be positive")
        canonical_dtype_name(self.dtype)
        _need(len(self.layers) > 0, "layers must name at least one layer")
        checks = dict(zip(TYPES, (_check_delta, _check_latent, _check_attention)))
        for i, layer in enumerate(self.layers):
            what = f"layers[{i}]"
            _keys(layer, {"type", "mixer"}, what, optional={"mlp"})
            _need(layer["type"] in checks,
                  f"{what}.type {layer['type']!r} is not known ({', '.join(TYPES)})")
            checks[layer["type"]](layer["mixer"], f"{what}.mixer")
            mlp = layer.get("mlp")
            if mlp is not None:
                _keys(mlp, {"kind", "ff"}, f"{what}.mlp")
                _need(mlp["kind"] == "dense", f"{what}.mlp.kind must be 'dense', got {mlp['kind']!r}")
                _positive_int(mlp["ff"], f"{what}.mlp.ff")
        mixing = self.mixing_layers()
        values = {(self.layers[i]["mixer"]["kv_heads"], self.layers[i]["mixer"]["vdim"])
                  for i in mixing}
        _need(len(values) <= 1, "layers with v_mix must have the same kv_heads and vdim, "
                                f"got {sorted(values)}")

    def mixing_layers(self) -> list:
        """The attention layers that mix their values, the one that fills them first."""
        return [i for i, layer in enumerate(self.layers)
                if layer["type"] == "attention" and layer["mixer"].get("v_mix")]

    @classmethod
    def from_dict(cls, raw: dict) -> "NekedraConfig":
        known = {"architecture", "vocab", "width", "layers", "norm", "max_seq_len", "dtype"}
        unknown = sorted(set(raw) - known)
        _need(not unknown, f"config.json has keys this architecture does not know: {unknown}")
        for req in ("vocab", "width", "layers", "norm"):
            _need(req in raw, f"config.json lacks the required key {req!r}")
        _keys(raw["norm"], {"eps"}, "norm")
        _need(isinstance(raw["layers"], list), "layers must be a list")
        return cls(architecture=raw.get("architecture", "Nekedra"), vocab=raw["vocab"],
                   width=raw["width"], layers=tuple(raw["layers"]),
                   norm_eps=_positive(raw["norm"]["eps"], "norm.eps"),
                   max_seq_len=raw.get("max_seq_len", DEFAULT_MAX_SEQ_LEN),
                   dtype=canonical_dtype_name(raw.get("dtype", "bfloat16")))

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "layers": list(self.layers),
               "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}
        if self.max_seq_len != DEFAULT_MAX_SEQ_LEN:
            out["max_seq_len"] = self.max_seq_len
        if self.dtype != "bfloat16":
            out["dtype"] = self.dtype
        return out
