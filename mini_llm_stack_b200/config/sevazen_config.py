"""Typed configuration of the Sevazen decoder, read from its config.json.

config.json: ``architecture``, ``vocab``, ``width``, ``norm.eps`` and ``layers``, a list in which
every entry names its mixer (``type``: ``attention`` or ``attention_2``), the mixer's sizes and
constants (``mixer``), its feed-forward (``mlp``, or null for none) and maybe another layer whose
tensors it uses (``weights_of``; the rest of the entry then equals that layer's).

* both mixers: ``heads``, ``kv_heads``, ``dim`` (queries and keys; of one map in ``attention_2``),
  ``vdim``, ``scale``, ``mask.size`` and ``rot`` (``base``, ``dims``, ``scaling``); ``mask``, ``rot``
  and ``rot.scaling`` may be null or absent: no limit, no rotation, plain frequencies.
* ``attention``: windows of ``mask.size`` tokens; ``conv`` taps of the short convolutions (null or
  absent: none); ``rot.scaling`` has ``factor``, ``low``, ``high`` and ``original``.
* ``attention_2``: chunks of ``mask.size`` tokens; ``diff``; ``rot.scaling`` has ``factor``,
  ``original``, ``fast`` and ``slow``.
* ``mlp``: ``kind`` ``dense`` with ``ff``, or ``moe`` with ``router`` (``experts``, ``top``),
  ``expert.ff`` and maybe ``shared.ff``.

Every size and constant of a model comes from there.  Positions are not bounded by a table, so
a sequence is as long as the engine lets it be (``max_seq_len``, an engine-side bound that
config.json may carry).
"""

from __future__ import annotations

from dataclasses import dataclass

from .model_config import ConfigError, canonical_dtype_name

DEFAULT_MAX_SEQ_LEN = 1 << 20
SCALING = {"attention": ("factor", "low", "high", "original"),
           "attention_2": ("factor", "original", "fast", "slow")}


def _need(cond, msg):
    if not cond:
        raise ConfigError(msg)


def _positive_int(v, what):
    _need(isinstance(v, int) and not isinstance(v, bool) and v > 0,
          f"{what} must be a positive integer, got {v!r}")
    return v


def _number(v, what):
    _need(isinstance(v, (int, float)) and not isinstance(v, bool), f"{what} must be a number, got {v!r}")
    return float(v)


def _positive(v, what):
    _need(_number(v, what) > 0, f"{what} must be a positive number, got {v!r}")
    return float(v)


def _keys(d, want: set, what: str, optional: set = frozenset()):
    _need(isinstance(d, dict), f"{what} must be an object, got {d!r}")
    missing, unknown = want - set(d), set(d) - want - optional
    _need(not missing, f"{what} lacks {sorted(missing)}")
    _need(not unknown, f"{what} has keys this architecture does not know: {sorted(unknown)}")


def _check_rotation(rot, dim: int, names, what: str) -> None:
    _keys(rot, {"base", "dims"}, what, optional={"scaling"})
    base = _positive(rot["base"], f"{what}.base")
    dims = _positive_int(rot["dims"], f"{what}.dims")
    _need(dims % 2 == 0 and dims <= dim, f"{what}.dims ({dims}) must be even and at most dim ({dim})")
    scaling = rot.get("scaling")
    if scaling is None:
        return
    _keys(scaling, set(names), f"{what}.scaling")
    for n in names:
        _positive(scaling[n], f"{what}.scaling.{n}")
    if "low" in names:
        _need(scaling["low"] != scaling["high"], f"{what}.scaling.low and .high must differ")
    else:
        _need(base != 1, f"{what}.base must not be 1 with this scaling")


def _check_mixer(kind: str, m, what: str) -> None:
    names = ("dim", "heads", "kv_heads", "vdim")
    own = {"diff"} if kind == "attention_2" else set()
    optional = {"mask", "rot"} | ({"conv"} if kind == "attention" else set())
    _keys(m, {*names, "scale"} | own, what, optional=optional)
    for n in names:
        _positive_int(m[n], f"{what}.{n}")
    _need(m["heads"] % m["kv_heads"] == 0,
          f"{what}.heads ({m['heads']}) must be a multiple of kv_heads ({m['kv_heads']})")
    _number(m["scale"], f"{what}.scale")
    if own:
        _number(m["diff"], f"{what}.diff")
    if m.get("conv") is not None:
        _positive_int(m["conv"], f"{what}.conv")
    if m.get("mask") is not None:
        _keys(m["mask"], {"size"}, f"{what}.mask")
        _positive_int(m["mask"]["size"], f"{what}.mask.size")
    if m.get("rot") is not None:
        _check_rotation(m["rot"], m["dim"], SCALING[kind], f"{what}.rot")


def _check_mlp(mlp, what: str) -> None:
    _need(isinstance(mlp, dict) and mlp.get("kind") in ("dense", "moe"),
          f"{what}.kind must be 'dense' or 'moe', got {mlp!r}")
    if mlp["kind"] == "dense":
        _keys(mlp, {"kind", "ff"}, what)
        _positive_int(mlp["ff"], f"{what}.ff")
        return
    _keys(mlp, {"kind", "expert", "router"}, what, optional={"shared"})
    _keys(mlp["expert"], {"ff"}, f"{what}.expert")
    _positive_int(mlp["expert"]["ff"], f"{what}.expert.ff")
    _keys(mlp["router"], {"experts", "top"}, f"{what}.router")
    experts = _positive_int(mlp["router"]["experts"], f"{what}.router.experts")
    top = _positive_int(mlp["router"]["top"], f"{what}.router.top")
    _need(top <= experts, f"{what}.router.top ({top}) must be at most experts ({experts})")
    if mlp.get("shared") is not None:
        _keys(mlp["shared"], {"ff"}, f"{what}.shared")
        _positive_int(mlp["shared"]["ff"], f"{what}.shared.ff")


@dataclass(frozen=True)
class SevazenConfig:
    architecture: str = "Sevazen"
    vocab: int = 256
    width: int = 64
    layers: tuple = ()
    norm_eps: float = 1e-5
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
        for i, layer in enumerate(self.layers):
            what = f"layers[{i}]"
            _keys(layer, {"type", "mixer"}, what, optional={"mlp", "weights_of"})
            _need(layer["type"] in SCALING,
                  f"{what}.type {layer['type']!r} is not known ({', '.join(SCALING)})")
            _check_mixer(layer["type"], layer["mixer"], f"{what}.mixer")
            if layer.get("mlp") is not None:
                _check_mlp(layer["mlp"], f"{what}.mlp")
            other = layer.get("weights_of")
            if other is not None:
                _need(isinstance(other, int) and not isinstance(other, bool)
                      and 0 <= other < len(self.layers) and other != i,
                      f"{what}.weights_of must name another layer, got {other!r}")
        for i, layer in enumerate(self.layers):
            mine, theirs = ({k: v for k, v in self.layers[j].items()
                             if k != "weights_of" and v is not None} for j in (i, self.owner(i)))
            _need(mine == theirs, f"layers[{i}].weights_of: the rest of the entry must equal layer "
                                  f"{self.owner(i)}'s")

    def owner(self, i: int) -> int:
        """The layer whose tensors layer ``i`` uses (itself, without ``weights_of``)."""
        seen = {i}
        while self.layers[i].get("weights_of") is not None:
            i = self.layers[i]["weights_of"]
            _need(i not in seen, f"layers[{i}].weights_of leads back to the layer itself")
            seen.add(i)
        return i

    @classmethod
    def from_dict(cls, raw: dict) -> "SevazenConfig":
        known = {"architecture", "vocab", "width", "layers", "norm", "max_seq_len", "dtype"}
        unknown = sorted(set(raw) - known)
        _need(not unknown, f"config.json has keys this architecture does not know: {unknown}")
        for req in ("vocab", "width", "layers", "norm"):
            _need(req in raw, f"config.json lacks the required key {req!r}")
        _keys(raw["norm"], {"eps"}, "norm")
        _need(isinstance(raw["layers"], list), "layers must be a list")
        return cls(architecture=raw.get("architecture", "Sevazen"), vocab=raw["vocab"],
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
