"""Tiny Sevazen configurations and helpers for the tests.

Sizes are chosen so that nothing the engine could confuse is equal: query/key and value sizes, head
counts and group sizes differ between layers; head sizes fall on and off the kernels' multiples
of 16 and on both sides of 32 and 64; one, two, three, four, five and nine taps and none; windows
and chunks of one token, shorter than a page, a page long, between pages, longer than the prompts,
absent; rotations of a part of a head, of a whole head, of none, with and without scaling; routers
that take one, some or all experts, with and without a shared expert; layers without feed-forward;
layers that use an earlier or a later layer's tensors; widths that are no multiple of eight.
"""

import json
from pathlib import Path

import torch
from safetensors.torch import save_file

from mini_llm_stack_b200.config import config_from_dict
from mini_llm_stack_b200.weights import random_tensors


def bands(factor, low, high, original):
    return {"factor": factor, "high": high, "low": low, "original": original}


def yarn(factor, original, fast, slow):
    return {"factor": factor, "fast": fast, "original": original, "slow": slow}


def rot(dims, base, scaling=None):
    out = {"base": base, "dims": dims}
    if scaling is not None:
        out["scaling"] = scaling
    return out


def _mixer(kind, heads, kv_heads, dim, vdim, scale, size, rotation, **more):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": vdim}
    if size is not None:
        m["mask"] = {"size": size}
    if rotation is not None:
        m["rot"] = rotation
    m.update({k: v for k, v in more.items() if v is not None})
    return {"type": kind, "mixer": m}


def window(heads, kv_heads, dim, vdim, scale, size=None, rotation=None, conv=None):
    return _mixer("attention", heads, kv_heads, dim, vdim, scale, size, rotation, conv=conv)


def pair(heads, kv_heads, dim, vdim, scale, diff, size=None, rotation=None):
    return _mixer("attention_2", heads, kv_heads, dim, vdim, scale, size, rotation, diff=diff)


def dense(ff):
    return {"ff": ff, "kind": "dense"}


def moe(experts, top, ff, shared=None):
    out = {"expert": {"ff": ff}, "kind": "moe", "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def layer(mixer, mlp=None):
    return dict(mixer, mlp=mlp)


def again(layers, of):
    """A layer with the tensors of ``layers[of]``."""
    return dict(layers[of], weights_of=of)


def model(layers, width=40, vocab=61, eps=1e-5) -> dict:
    return {"architecture": "Sevazen", "layers": layers, "norm": {"eps": eps}, "vocab": vocab,
            "width": width}


def _mixed():
    layers = [
        layer(window(6, 3, 12, 20, 0.3, 19, rot(8, 300.0, bands(4.0, 1.0, 4.0, 64)), 3), moe(7, 3, 12, 20)),
        layer(pair(4, 2, 8, 12, 0.35, 0.3, 24, rot(6, 100.0, yarn(8.0, 256, 8.0, 1.0))), dense(28)),
        layer(window(4, 4, 20, 8, 0.25, 33, rot(20, 1000.0), 5)),
        layer(pair(3, 1, 10, 24, 0.3, 0.5, 37, rot(10, 50.0, yarn(2.0, 128, 16.0, 2.0))), moe(5, 5, 8)),
    ]
    layers.append(again(layers, 0))
    layers.append(again(layers, 1))
    layers.append(again(layers, 0))
    return model(layers, width=44, vocab=97)


# every mechanism, nothing equal to anything else; shared tensors with caches and tails of their own
S_MIXED = _mixed()

# the pieces that may be absent: no mask, no rotation, no scaling, no convolution, one tap, one
# expert of one, no shared expert, no feed-forward; a window and a chunk of one token; a layer that
# uses the tensors of a later one; a width that is no multiple of four
S_BARE = model([
    layer(window(2, 1, 10, 6, 0.4), moe(1, 1, 10)),
    dict(layer(pair(2, 2, 6, 6, 0.4, 0.2, 16, rot(2, 30.0)), dense(12)), weights_of=3),
    layer(window(3, 1, 16, 16, 0.3, 1, None, 1), moe(6, 1, 8, 14)),
    layer(pair(2, 2, 6, 6, 0.4, 0.2, 16, rot(2, 30.0)), dense(12)),
    layer(pair(5, 5, 7, 9, 0.3, 0.8, None, None)),
    layer(window(2, 2, 5, 34, 0.5, 16, rot(4, 1e4, bands(2.0, 0.5, 2.0, 40)), 9), dense(16)),
    layer(pair(1, 1, 16, 32, 0.3, 0.1, 1, rot(16, 200.0)), moe(4, 2, 6, 6)),
], width=38, vocab=53, eps=1e-6)

# head sizes of 64 and 128: the sizes at which the bfloat16 run takes its tensor-core paths;
# groups of 2 x 12 query rows a cached head
S_WIDE = model([
    layer(window(4, 2, 64, 64, 0.125, 48, rot(32, 1e4, bands(8.0, 1.0, 4.0, 128)), 4), dense(160)),
    layer(pair(6, 3, 32, 64, 0.18, 0.4, 80, rot(16, 1e4, yarn(4.0, 512, 32.0, 1.0))), moe(8, 2, 64, 96)),
    layer(window(2, 1, 128, 96, 0.09, 100, rot(128, 5e4, bands(4.0, 1.0, 4.0, 200)), 2), moe(6, 3, 40)),
    layer(pair(12, 1, 48, 128, 0.14, 0.2, 64, rot(48, 1e4)), dense(96)),
], width=128, vocab=131, eps=1e-6)


def one_layer(mixer_layer, mlp=None, **top) -> dict:
    """A model of the embedding, one layer, the final norm and the tied head."""
    return model([layer(mixer_layer, mlp)], **top)


def sharp(factor):
    """Scale the query norms' weights so that a softmax picks nearly one key."""
    def patch(w):
        for n in w:
            if n.endswith("mix.q.norm"):
                w[n] *= factor
    return patch


def decisive_routers(w):
    """Routers whose choices rest on their biases: every logit lies far from the next, in an order
    of its own; the chosen experts' weights still follow the tokens."""
    for n in w:
        if n.endswith("router.b"):
            order = torch.randperm(w[n].numel(), generator=torch.Generator().manual_seed(len(n)))
            w[n] = 0.5 * order.float()
        if n.endswith("mlp.router"):
            w[n] *= 0.02


def make_sevazen(folder, raw: dict, seed: int, dtype: str = "bfloat16", std: float = 0.15,
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
        elif last == "sink":
            t = draw
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            t = draw * 0.3
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
