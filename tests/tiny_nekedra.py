"""Tiny Nekedra configurations and helpers for the tests.

Sizes are chosen so that nothing the engine could confuse is equal: key and value sizes, head
counts and group sizes differ between layers; head sizes fall on and off the kernels' multiples
of 16 and 32; latents plus rotated parts fall on and off the attention kernels' sizes;
convolutions have one, two, three, four, five and nine taps; attention layers mix their values,
fill them or stand apart; layers have no feed-forward; a width is no multiple of eight.
"""

import json
from pathlib import Path

import torch
from safetensors.torch import save_file

from mini_llm_stack_b200.config import config_from_dict
from mini_llm_stack_b200.weights import random_tensors


def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "delta", "mixer": {"conv": conv, "dim": dim, "heads": heads,
                                       "kv_heads": kv_heads, "vdim": vdim}}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=1000.0):
    return {"type": "latent_attention",
            "mixer": {"dim": dim, "heads": heads, "kv_rank": kv_rank,
                      "rot": {"base": base, "dims": rot_dim}, "rot_dim": rot_dim, "scale": scale,
                      "vdim": vdim}}


def attention(heads, kv_heads, dim, vdim, scale, v_mix=None):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": vdim}
    if v_mix is not None:
        m["v_mix"] = v_mix
    return {"type": "attention", "mixer": m}


def layer(mixer, ff=None):
    return dict(mixer, mlp=None if ff is None else {"ff": ff, "kind": "dense"})


def model(layers, width=40, vocab=61, eps=1e-5) -> dict:
    return {"architecture": "Nekedra", "layers": layers, "norm": {"eps": eps}, "vocab": vocab,
            "width": width}


# every mechanism, nothing equal to anything else; the layer that fills the values is not the
# first layer, and an attention layer between two mixing ones stands apart
N_MIXED = model([
    layer(delta(4, 2, 12, 20, 3), 24),
    layer(attention(4, 2, 12, 20, 0.3, v_mix=True), 32),
    layer(latent(3, 10, 6, 14, 18, 0.25), 20),
    layer(attention(3, 3, 16, 8, 0.2, v_mix=False)),
    layer(delta(3, 3, 40, 8, 4)),
    layer(attention(6, 2, 8, 20, 0.35, v_mix=True), 28),
    layer(attention(2, 2, 24, 20, 0.15, v_mix=True), 16),
], width=40, vocab=97)

# no value mixing; attention first, a width that is no multiple of eight, a convolution of one
# tap and one of nine, one key head for all value heads, a head count that is no multiple of four
N_PLAIN = model([
    layer(attention(2, 1, 10, 6, 0.4), 12),
    layer(delta(5, 1, 6, 10, 1), 20),
    layer(latent(5, 4, 2, 6, 10, 0.5, base=50.0)),
    layer(delta(2, 2, 34, 18, 9)),
], width=36, vocab=53, eps=1e-6)

# head sizes of 64 and 128: the sizes at which the bfloat16 run takes its tensor-core paths
N_WIDE = model([
    layer(delta(4, 2, 64, 128, 4), 160),
    layer(attention(4, 2, 64, 64, 0.125, v_mix=True), 96),
    layer(latent(4, 48, 32, 40, 96, 0.11, base=1e5), 128),
    layer(attention(2, 2, 48, 64, 0.14, v_mix=True)),
    layer(delta(2, 1, 128, 48, 2), 64),
], width=128, vocab=131, eps=1e-6)


def one_layer(mixer_layer, ff=None, **top) -> dict:
    """A model of the embedding, one layer, the final norm and the head."""
    return model([layer(mixer_layer, ff)], **top)


def sharp(factor):
    """Scale the attention layers' queries so that a softmax picks nearly one key."""
    def patch(w):
        for n in w:
            kind = n.split(".")
            if kind[-2:] == ["mix", "q"] and f"{kind[0]}.mix.q.conv" not in w:
                w[n] *= factor
            if n.endswith("mix.q.b"):
                w[n] *= factor
    return patch


def slow_decay(w):
    """Decays close to one: what enters the state stays for hundreds of tokens."""
    for n in w:
        if n.endswith("A_log"):
            w[n] -= 5.0


def make_nekedra(folder, raw: dict, seed: int, dtype: str = "bfloat16", std: float = 0.15,
                 patch=None):
    """Write a model folder; returns the config as stored and float64 numpy weights as the
    file holds them.  Matrices are drawn with a larger deviation than the engine's default so
    that every mechanism moves the logits; ``patch(weights)`` may change tensors before they are
    stored (in the stored dtype's rounding)."""
    cfg = config_from_dict(dict(raw, dtype=dtype))
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    g = torch.Generator().manual_seed(seed + 1000)
    w = {}
    for name, t in random_tensors(cfg, seed, 0.0, dtype="float32"):
        last = name.rsplit(".", 1)[-1]
        draw = torch.randn(t.shape, generator=g)
        if last == "conv":
            t = draw * 0.5
        elif last in ("sink", "dt_bias", "A_log"):
            t = draw
        elif last == "vmix":
            t = 0.4 + 0.1 * draw
        elif last == "b" and t.dim() == 1:
            t = draw * 0.5
        elif t.dim() <= 1:
            t = 1.0 + 0.2 * draw                       # norm weights
        elif name == "embed":
            t = draw
        else:
            t = draw * std
        w[name] = t
    if patch:
        patch(w)
    store = torch.bfloat16 if dtype == "bfloat16" else torch.float32
    w = {n: t.to(store).contiguous() for n, t in w.items()}
    save_file(w, str(folder / "model.safetensors"))
    stored = cfg.to_dict()
    (folder / "config.json").write_text(json.dumps(stored, indent=1))
    return stored, {n: t.double().numpy() for n, t in w.items()}
