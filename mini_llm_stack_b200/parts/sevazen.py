"""Sevazen: layers of windowed attention with sinks behind short convolutions, or of differential
attention within chunks, each followed by a dense ungated unit, routed ungated experts or nothing;
layer norms behind the sublayers only, layers that share another's tensors, a tied output head.

Tensor names: ``embed``, ``l<i>.norm1 / norm2`` (and ``.b``), ``l<i>.mix.*``, ``l<i>.mlp.*``,
``final.norm`` (and ``.b``).  A layer with the tensors of another is another call of that layer's
block, with a cache slot of its own.
"""

from __future__ import annotations

from ..config.registry import register_architecture
from ..config.sevazen_config import SevazenConfig
from .attention import DifferentialAttention, RotatedAttention
from .block import PostNormBlock
from .feedforward import RoutedExperts, SquaredReluFeedForward
from .model import ComposedModel, LayerCall, OutputHead, TokenEmbedding
from .norm import LayerNorm
from .position import BandScaling, PartialRotary, YarnScaling


def _rotary(rot, scaling_class):
    if rot is None:
        return None
    scaling = rot.get("scaling")
    return PartialRotary(rot["dims"], rot["base"], pairing="half",
                         scaling=scaling_class(**scaling) if scaling is not None else None)


def _mixer(cfg: SevazenConfig, layer: dict):
    m = layer["mixer"]
    span = (m.get("mask") or {}).get("size")
    sizes = (cfg.width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], cfg.norm_eps)
    if layer["type"] == "attention":
        return RotatedAttention(*sizes, position=_rotary(m.get("rot"), BandScaling),
                                taps=m.get("conv") or 0, window=span, sink=True)
    return DifferentialAttention(*sizes, m["diff"], position=_rotary(m.get("rot"), YarnScaling),
                                 chunk=span)


def _feedforward(cfg: SevazenConfig, mlp):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return SquaredReluFeedForward(cfg.width, mlp["ff"])
    shared = None
    if mlp.get("shared") is not None:
        shared = SquaredReluFeedForward(cfg.width, mlp["shared"]["ff"])
    router = mlp["router"]
    return RoutedExperts(cfg.width, router["experts"], router["top"], mlp["expert"]["ff"],
                         shared=shared, weigh="output", score="logit", router_bias=True,
                         shared_gate=shared is not None, unit="relu_squared")


def build_sevazen(cfg: SevazenConfig) -> ComposedModel:
    def norm():
        return LayerNorm(cfg.width, cfg.norm_eps, tensor_name="", bias=True)

    owners = [i for i in range(len(cfg.layers)) if cfg.owner(i) == i]
    blocks = []
    for i in owners:
        ffn = _feedforward(cfg, cfg.layers[i].get("mlp"))
        blocks.append(PostNormBlock(_mixer(cfg, cfg.layers[i]), norm(), ffn,
                                    norm() if ffn is not None else None, cfg.width))
    calls = [LayerCall(owners.index(cfg.owner(i)), i) for i in range(len(cfg.layers))]
    embedding = TokenEmbedding(cfg.vocab, cfg.width, tensor_name="")
    return ComposedModel(cfg, embedding, blocks, calls, norm(),
                         OutputHead(cfg.vocab, cfg.width, tied_to=embedding),
                         names=("embed", None, "final.norm", None),
                         block_prefix=lambda k: f"l{owners[k]}")


register_architecture("Sevazen", SevazenConfig, build_sevazen, aliases=("sevazen",))
