"""Nekedra: layers of the gated delta rule, of latent attention with a rotated key part and one
gate a head, and of unrotated attention with sinks whose later layers mix their values with the
first such layer's; RMS norms of one number before and behind every sublayer, a full sigmoid
gate on every sublayer's result, dense gated units, an untied output head.

Tensor names: ``embed``, ``l<i>.norm1 / norm1b / norm2 / norm2b``, ``l<i>.rg1 / rg2`` (and ``.b``),
``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from ..config.nekedra_config import NekedraConfig
from ..config.registry import register_architecture
from .attention import FirstValues, UnrotatedAttention
from .block import GatedSandwichBlock
from .feedforward import SwiGLUFeedForward
from .latent_attention import RotaryLatentAttention
from .linear_recurrence import GatedDeltaMixer
from .model import ComposedModel, LayerCall, OutputHead, TokenEmbedding
from .norm import RMSNorm
from .position import PartialRotary


def _mixer(cfg: NekedraConfig, index: int, mixing: list, first_values):
    m, kind = cfg.layers[index]["mixer"], cfg.layers[index]["type"]
    if kind == "delta":
        return GatedDeltaMixer(cfg.width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"],
                               cfg.norm_eps)
    if kind == "latent_attention":
        return RotaryLatentAttention(
            cfg.width, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"],
            cfg.norm_eps, sink=False, gate="head",
            position=PartialRotary(m["rot"]["dims"], m["rot"]["base"], 1.0, "interleaved"))
    return UnrotatedAttention(
        cfg.width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], cfg.norm_eps,
        qkv_bias=True, sink=True, first_values=first_values if index in mixing else None,
        fills_first=index == (mixing[0] if mixing else -1))


def build_nekedra(cfg: NekedraConfig) -> ComposedModel:
    def norm():
        return RMSNorm(cfg.width, cfg.norm_eps, tensor_name="", scalar=True)

    mixing, first_values = cfg.mixing_layers(), None
    if mixing:
        m = cfg.layers[mixing[0]]["mixer"]
        first_values = FirstValues(m["kv_heads"], m["vdim"])
    blocks, calls = [], []
    for i, layer in enumerate(cfg.layers):
        mlp = layer.get("mlp")
        ffn = (SwiGLUFeedForward(cfg.width, mlp["ff"], names=("gate", "up", "down"))
               if mlp is not None else None)
        blocks.append(GatedSandwichBlock(norm(), _mixer(cfg, i, mixing, first_values), norm(),
                                         norm() if ffn is not None else None, ffn,
                                         norm() if ffn is not None else None, cfg.width))
        calls.append(LayerCall(i, i, writes=True))
    return ComposedModel(cfg, TokenEmbedding(cfg.vocab, cfg.width, tensor_name=""), blocks, calls,
                         norm(), OutputHead(cfg.vocab, cfg.width, tied_to=None, tensor_name=""),
                         names=("embed", None, "final.norm", "head"),
                         block_prefix=lambda i: f"l{i}")


register_architecture("Nekedra", NekedraConfig, build_nekedra, aliases=("nekedra",))
