"""The arrangement of a layer's parts: the pre-norm residual block, the block with a norm before
and behind every sublayer, that block with a gate on every sublayer's result, and the block with
norms behind the sublayers only.

Reference (train/model.py:200-217): ``x = x + mixer(norm_a(x))``;
``x = x + feed_forward(norm_b(x))``.  The block owns the order and the names
its parts' tensors carry in a weight file; the parts own the math.
"""

from __future__ import annotations

import torch

from .base import CacheHandle, Part, ResidualStream, StepContext, TensorSpec
from .norm import StreamRows


def join_name(prefix: str, name: str) -> str:
    """``prefix.name``; an empty ``name`` is the prefix itself (a part whose one tensor
    carries the part's own name)."""
    if not name:
        return prefix
    return f"{prefix}.{name}" if prefix else name


def under_prefix(tensors: dict, prefix: str) -> dict:
    """The tensors of ``prefix`` under their local names (``prefix`` itself becomes "")."""
    out = {}
    for n, t in tensors.items():
        if n == prefix:
            out[""] = t
        elif n.startswith(prefix + "."):
            out[n[len(prefix) + 1:]] = t
    return out


class PreNormBlock(Part):
    tail = None

    def __init__(self, mixer_norm, mixer, ffn_norm, ffn,
                 names=("attn_norm", "attn", "mlp_norm", "mlp"), tail=None):
        """``tail``: a part that runs last, on the stream itself (``forward(stream, step)``:
        it settles what is pending and pushes its own delta); its prefix is a fifth name."""
        self.mixer_norm, self.mixer = mixer_norm, mixer
        self.ffn_norm, self.ffn = ffn_norm, ffn
        self.tail = tail
        self.names = tuple(names)
        if tail is not None and len(self.names) < 5:
            raise ValueError("a block with a tail needs a fifth name, the tail's prefix")

    def _named_parts(self):
        """(prefix, part) of the parts there are; a block without a feed-forward
        (``ffn`` None) has no second norm either."""
        return [(n, p) for n, p in zip(self.names, (self.mixer_norm, self.mixer,
                                                    self.ffn_norm, self.ffn, self.tail))
                if p is not None]

    def tensor_specs(self) -> dict:
        out = {}
        for prefix, part in self._named_parts():
            for n, s in part.tensor_specs().items():
                out[join_name(prefix, n)] = s
        return out

    def bind(self, tensors: dict, runtime) -> None:
        self.runtime = runtime
        for prefix, part in self._named_parts():
            part.bind(under_prefix(tensors, prefix), runtime)

    def cache_spec(self):
        return self.mixer.cache_spec()

    @property
    def decode_capturable(self) -> bool:
        return all(getattr(p, "decode_capturable", False) for _, p in self._named_parts())

    @property
    def prompt_capturable(self) -> bool:
        return all(getattr(p, "prompt_capturable", False) for _, p in self._named_parts())

    def decode_graph_key(self, step: StepContext) -> tuple:
        return tuple(k for _, p in self._named_parts() if (k := p.decode_graph_key(step)))

    def forward(self, stream: ResidualStream, step: StepContext,
                cache: CacheHandle) -> None:
        h = self.mixer_norm.forward(stream)
        delta = self.mixer.forward(h, step, cache)
        if isinstance(delta, tuple):
            # (delta, a vector for every row): a mixer whose output projection has a bias
            delta, vec = delta
            stream.push_more(vec=vec)
        stream.push(delta)
        if self.ffn is not None:
            h = self.ffn_norm.forward(stream)
            stream.push(self.ffn.forward(h, step))
        if self.tail is not None:
            self.tail.forward(stream, step)


class SandwichBlock(PreNormBlock):
    """A norm before and behind each sublayer, and an optional per-channel scale on what
    joins the stream: ``x <- x + s1 * post1(mixer(pre1(x)))``; ``x <- x + s2 *
    post2(ffn(pre2(x)))``.  The norms behind the sublayers are of a kind that can ride on the
    pending delta (``norm.mapped(delta, scale, bias)``, e.g. ``DynamicTanhNorm``): they cost
    no pass of their own.  A sublayer may return ``(delta, vector)``: the vector (an output
    bias) is added to every row before the norm behind it.

    ``names``: prefixes of (pre1, mixer, post1, pre2, ffn, post2); ``scale_names``: the two
    scale vectors' tensor names, or None for a block without them."""

    def __init__(self, mixer_norm, mixer, mixer_post, ffn_norm, ffn, ffn_post, d_model: int,
                 names=("norm1", "mix", "norm1b", "norm2", "mlp", "norm2b"),
                 scale_names=("ls1", "ls2")):
        self.mixer_norm, self.mixer, self.mixer_post = mixer_norm, mixer, mixer_post
        self.ffn_norm, self.ffn, self.ffn_post = ffn_norm, ffn, ffn_post
        self.d_model = int(d_model)
        self.names, self.scale_names = tuple(names), scale_names
        self.scales = [None, None]

    def _named_parts(self):
        parts = (self.mixer_norm, self.mixer, self.mixer_post, self.ffn_norm, self.ffn,
                 self.ffn_post)
        return [(n, p) for n, p in zip(self.names, parts) if p is not None]

    def tensor_specs(self) -> dict:
        out = super().tensor_specs()
        if self.scale_names is not None:
            out[self.scale_names[0]] = TensorSpec((self.d_model,), kind="vector", init="ones")
            if self.ffn is not None:
                out[self.scale_names[1]] = TensorSpec((self.d_model,), kind="vector", init="ones")
        return out

    def bind(self, tensors: dict, runtime) -> None:
        super().bind(tensors, runtime)
        if self.scale_names is not None:
            self.scales = [tensors[n].contiguous() if n in tensors else None
                           for n in self.scale_names]

    @staticmethod
    def _push(stream: ResidualStream, post, out, scale) -> None:
        bias = None
        if isinstance(out, tuple):
            out, bias = out
        stream.push(post.mapped(out, scale, bias))

    def forward(self, stream: ResidualStream, step: StepContext, cache: CacheHandle) -> None:
        h = self.mixer_norm.forward(stream)
        self._push(stream, self.mixer_post, self.mixer.forward(h, step, cache), self.scales[0])
        if self.ffn is None:
            return
        h = self.ffn_norm.forward(stream)
        self._push(stream, self.ffn_post, self.ffn.forward(h, step), self.scales[1])


class GatedSandwichBlock(SandwichBlock):
    """A norm before and behind each sublayer and a full gate on its result: with
    ``h = pre(x)``, ``x <- x + post(sublayer(h) * sigmoid(W h + b))`` for the mixer, then for the
    feed-forward.  The gate, the norm behind the sublayer, the sum and the next norm are one
    kernel (``RMSNorm.gated``).  The mixer's gate rides on the product that reads the mixer's
    input where the mixer allows it (``Mixer.takes_rider``); the feed-forward's is a product of
    its own whose K-parts may be left to that kernel.

    ``gate_names``: prefixes of the two gates' matrices; their biases carry ``.b`` behind it."""

    def __init__(self, mixer_norm, mixer, mixer_post, ffn_norm, ffn, ffn_post, d_model: int,
                 names=("norm1", "mix", "norm1b", "norm2", "mlp", "norm2b"),
                 gate_names=("rg1", "rg2")):
        super().__init__(mixer_norm, mixer, mixer_post, ffn_norm, ffn, ffn_post, d_model,
                         names=names, scale_names=None)
        self.gate_names = tuple(gate_names)
        self.gate_w, self.gate_b = [None, None], [None, None]

    def _gates(self):
        return self.gate_names if self.ffn is not None else self.gate_names[:1]

    def tensor_specs(self) -> dict:
        out = super().tensor_specs()
        d = self.d_model
        for n in self._gates():
            out[n] = TensorSpec((d, d))
            out[join_name(n, "b")] = TensorSpec((d,), kind="vector", init="zeros")
        return out

    def bind(self, tensors: dict, runtime) -> None:
        self.runtime = runtime
        self.gate_w, self.gate_b = [None, None], [None, None]
        for i, n in enumerate(self._gates()):
            self.gate_w[i] = tensors[n]
            self.gate_b[i] = tensors[join_name(n, "b")].float().contiguous()
        for prefix, part in self._named_parts():
            mine = under_prefix(tensors, prefix)
            if part is self.mixer and part.takes_rider:
                part.bind(mine, runtime, rider=self.gate_w[0])
                self.gate_w[0] = None
            else:
                part.bind(mine, runtime)
        self.gate_w = [None if w is None else runtime.ops.prepare_weight(w) for w in self.gate_w]
        runtime.ops.require_part("gatednorm")

    def _gate(self, i: int, h):
        """The gate's pre-activation as a product of its own (maybe left as its K-parts)."""
        rt = self.runtime
        z = rt.buffer("residual_gate", (h.shape[0], self.d_model), torch.float32)
        got = rt.ops.linear_parts(h, self.gate_w[i], z, lend="gate")
        return (z, 0) if got is z else got

    def forward(self, stream: ResidualStream, step: StepContext, cache: CacheHandle) -> None:
        h = self.mixer_norm.forward(stream)
        gate = self._gate(0, h) if self.gate_w[0] is not None else None
        y = self.mixer.forward(h, step, cache)
        if isinstance(y, tuple):
            raise TypeError("a mixer with an output bias does not fit a gated block")
        stream.push(self.mixer_post.gated(y, gate or self.mixer.rider(), self.gate_b[0]))
        if self.ffn is None:
            return
        h = self.ffn_norm.forward(stream)
        gate = self._gate(1, h)
        stream.push(self.ffn_post.gated(self.ffn.forward(h, step), gate, self.gate_b[1]))


class PostNormBlock(PreNormBlock):
    """Norms behind the sublayers only: ``x <- x + post1(mixer(x))``; ``x <- x + post2(ffn(x))``.
    The sublayers read the stream itself (``StreamRows``), and that read is the pass in which the
    sublayer before is normed and added: as many kernels as a pre-norm block has.  The norms are of
    a kind that can wait on the stream (``norm.behind(delta, bias)``, e.g. ``LayerNorm``).

    ``names``: prefixes of (mixer, its norm, ffn, its norm)."""

    def __init__(self, mixer, mixer_post, ffn, ffn_post, d_model: int,
                 names=("mix", "norm1", "mlp", "norm2")):
        self.mixer, self.mixer_post, self.ffn, self.ffn_post = mixer, mixer_post, ffn, ffn_post
        self.rows = StreamRows(d_model)
        self.names = tuple(names)

    def _named_parts(self):
        parts = (self.mixer, self.mixer_post, self.ffn, self.ffn_post)
        return [(n, p) for n, p in zip(self.names, parts) if p is not None]

    def bind(self, tensors: dict, runtime) -> None:
        super().bind(tensors, runtime)
        self.rows.bind({}, runtime)

    @staticmethod
    def _push(stream: ResidualStream, post, out) -> None:
        out, bias = out if isinstance(out, tuple) else (out, None)
        stream.push(post.behind(out, bias))

    def forward(self, stream: ResidualStream, step: StepContext, cache: CacheHandle) -> None:
        self._push(stream, self.mixer_post, self.mixer.forward(self.rows.forward(stream), step, cache))
        if self.ffn is not None:
            self._push(stream, self.ffn_post, self.ffn.forward(self.rows.forward(stream), step))
