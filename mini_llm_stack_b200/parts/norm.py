"""Norms: RMS norm with a learned weight (a vector or one number; also behind a sublayer, with a
gate on the sublayer's result), layer norm with a weight and maybe a bias (also behind a
sublayer), the norm without statistics (a scaled tanh with a weight and a bias), and, for layers
that read the stream itself, none.

Reference formula (train/model.py:29-33): ``xf = x.float()``;
``y = xf * rsqrt(mean(xf**2, -1) + eps)``; ``out = (y * w.float()).to(x.dtype)``.
eps sits inside the square root, added to the mean; the weight multiplies after
the normalisation; no bias.  All of it runs in float32 with one rounding at the
end.  The residual stream's pending addend is added in the same pass.
"""

from __future__ import annotations

import torch

from .base import Norm, ResidualStream, TensorSpec


class GatedDelta:
    """A sublayer's output that is still to be gated and normed before it joins the residual
    stream: ``norm(delta * sigmoid(gate + bias))``.  ``gate``: None, ``(rows, first column)``
    or ``SplitParts``.  A norm that knows the kind (``RMSNorm.forward``) does it in the pass in
    which it adds the delta; any other consumer gets the values through ``resolve()`` (one kernel
    of its own, float32)."""

    def __init__(self, delta, norm: "RMSNorm", gate=None, bias=None):
        self.delta, self.norm, self.gate, self.bias = delta, norm, gate, bias

    @property
    def shape(self):
        return self.delta.shape

    def release(self) -> None:
        for p in (self.delta, self.gate):
            if hasattr(p, "release"):
                p.release()

    def resolve(self):
        rt = self.norm.runtime
        t, d = self.delta.shape
        out = rt.buffer("gated_delta", (t, d), torch.float32)
        rt.ops.add_gated_norm(None, self.delta, self.gate, self.bias, self.norm.weight32, None,
                              self.norm.eps, None, y_out=out)
        return out

    def float(self):
        return self.resolve()


class RMSNorm(Norm):
    decode_capturable = prompt_capturable = True   # forward only launches kernels on the current stream

    def __init__(self, dim: int, eps: float, tensor_name: str = "weight", one_plus: bool = False,
                 scalar: bool = False):
        """``tensor_name``: the local name of the weight ("" = the part's own prefix).
        ``one_plus``: the weight is stored around zero and multiplies as ``1 + w`` (the sum is
        taken once, in float32, when the weight is bound).  ``scalar``: the weight is one number
        for all coordinates (a tensor without dimensions).

        Behind a sublayer the norm does not run by itself: ``gated(delta, gate, bias)`` wraps
        the sublayer's output, and the norm that adds it to the stream does all of it in one
        kernel."""
        self.dim = int(dim)
        self.eps = float(eps)
        self.tensor_name = tensor_name
        self.one_plus, self.scalar = bool(one_plus), bool(scalar)
        self.weight = self.weight32 = None

    def tensor_specs(self) -> dict:
        return {self.tensor_name: TensorSpec(() if self.scalar else (self.dim,), kind="vector",
                                             init="zeros" if self.one_plus else "ones")}

    def bind(self, tensors: dict, runtime) -> None:
        self.runtime = runtime
        w = tensors[self.tensor_name]
        w = w.float() + 1.0 if self.one_plus else w
        self.weight32 = w.float().reshape(-1).contiguous()
        self.weight = (w.reshape(1).expand(self.dim) if self.scalar else w).contiguous()

    def gated(self, delta, gate=None, bias=None) -> GatedDelta:
        """``delta`` (a tensor or ``SplitParts``) as what the gate, then this norm, make of it,
        for ``ResidualStream.push``."""
        self.runtime.ops.require_part("gatednorm")
        return GatedDelta(delta, self, gate, bias)

    def forward(self, stream: ResidualStream, rows=None, n_rows: int = 0):
        """Add the pending delta into the stream, return the normalised rows.

        With ``rows`` (int32 row indices) only those rows are read, summed and
        normalised: the output is [n_rows, dim] and the stream itself is left
        as it was.
        """
        rt = self.runtime
        more_rows, more_vec = stream.take_more()
        if more_rows is not None or more_vec is not None:
            # (also before picked rows: the addends go into every row of the stream)
            rt.ops.residual_add(stream.x, more_rows, more_vec)
        delta = stream.take_pending()
        if isinstance(delta, GatedDelta) and delta.norm.eps == self.eps:
            n = stream.x.shape[0] if rows is None else n_rows
            h = rt.buffer("normed" if rows is None else "normed_rows", (n, self.dim), rt.act_dtype)
            rt.ops.add_gated_norm(stream.x, delta.delta, delta.gate, delta.bias,
                                  delta.norm.weight32, self.weight32, self.eps, h, rows=rows,
                                  n_rows=n_rows)
            return h
        if rows is None:
            t = stream.x.shape[0]
            h = rt.buffer("normed", (t, self.dim), rt.act_dtype)
            rt.ops.add_rmsnorm(stream.x, delta, self.weight, self.eps, h)
        else:
            h = rt.buffer("normed_rows", (n_rows, self.dim), rt.act_dtype)
            rt.ops.gather_add_rmsnorm(stream.x, delta, rows, n_rows, self.weight,
                                      self.eps, h)
        return h


class NormedDelta:
    """A sublayer's output that is still to be layer-normed (plus ``bias``, a vector for every row,
    first) before it joins the residual stream.  ``settle_normed`` does it in the pass in which it
    adds the delta; any other consumer gets the values through ``resolve()`` (one kernel of its
    own, float32)."""

    def __init__(self, delta, norm: "LayerNorm", bias=None):
        self.delta, self.norm, self.bias = delta, norm, bias

    @property
    def shape(self):
        return self.delta.shape

    def release(self) -> None:
        if hasattr(self.delta, "release"):
            self.delta.release()

    def resolve(self):
        rt = self.norm.runtime
        out = rt.buffer("normed_delta", tuple(self.delta.shape), torch.float32)
        rt.ops.add_post_layernorm(None, self.delta, self.norm.vectors, self.norm.eps, None,
                                  bias=self.bias, y_out=out)
        return out

    def float(self):
        return self.resolve()


def settle_normed(rt, stream: ResidualStream, h, norm=None, rows=None, n_rows: int = 0) -> None:
    """Add what waits on the stream and leave the stream's rows (all, or ``rows``) in ``h``: as they
    are, or through ``norm``, a ``LayerNorm`` with a bias.  One kernel where a ``NormedDelta`` of
    the same eps waits, or nothing."""
    more_rows, more_vec = stream.take_more()
    delta = stream.take_pending()
    eps = norm.eps if norm is not None else None
    if isinstance(delta, NormedDelta) and (eps is None or eps == delta.norm.eps):
        y, post, bias, eps = delta.delta, delta.norm.vectors, delta.bias, delta.norm.eps
    else:
        if delta is not None:
            rt.ops.residual_add(stream.x, delta.float())
        y = post = bias = None
    if more_rows is not None or more_vec is not None:
        rt.ops.residual_add(stream.x, more_rows, more_vec)
    rt.ops.add_post_layernorm(stream.x, y, post, eps or 0.0, h, bias=bias,
                              norm=norm.vectors if norm is not None else None, rows=rows,
                              n_rows=n_rows)


class StreamRows(Norm):
    """In the place of a norm before a sublayer that reads the residual stream itself: adds what
    waits on the stream and gives its rows in the activations' type."""

    decode_capturable = prompt_capturable = True

    def __init__(self, dim: int):
        self.dim = int(dim)

    def bind(self, tensors: dict, runtime) -> None:
        self.runtime = runtime
        runtime.ops.require_part("layernorm")

    def forward(self, stream: ResidualStream, rows=None, n_rows: int = 0):
        rt = self.runtime
        n, name = (stream.x.shape[0], "normed") if rows is None else (n_rows, "normed_rows")
        h = rt.buffer(name, (n, self.dim), rt.act_dtype)
        settle_normed(rt, stream, h, rows=rows, n_rows=n_rows)
        return h


class LayerNorm(Norm):
    """``(x - mean) / sqrt(var + eps) * w (+ b)`` with the biased variance, in
    float32 with one rounding.  Adds the stream's pending delta and its other waiting
    addends (``ResidualStream.push_more``) in the same pass.  ``tensor_name`` is the
    local name of the weight ("" = the part's own prefix); with ``bias`` the tensor ``b`` lies
    beside it.

    Behind a sublayer (a norm with a bias only) it does not run by itself: ``behind(delta,
    bias)`` wraps the sublayer's output, and what adds that to the stream norms it."""

    decode_capturable = prompt_capturable = True

    def __init__(self, dim: int, eps: float, tensor_name: str = "weight", bias: bool = False):
        self.dim, self.eps, self.tensor_name = int(dim), float(eps), tensor_name
        self.has_bias = bool(bias)
        self.weight = self.vectors = None

    def _bias_name(self) -> str:
        return f"{self.tensor_name}.b" if self.tensor_name else "b"

    def tensor_specs(self) -> dict:
        out = {self.tensor_name: TensorSpec((self.dim,), kind="vector", init="ones")}
        if self.has_bias:
            out[self._bias_name()] = TensorSpec((self.dim,), kind="vector", init="zeros")
        return out

    def bind(self, tensors: dict, runtime) -> None:
        self.runtime = runtime
        self.weight = tensors[self.tensor_name].contiguous()
        if self.has_bias:
            self.vectors = (self.weight.float().contiguous(),
                            tensors[self._bias_name()].float().contiguous())
        runtime.ops.require_part("layernorm")

    def behind(self, delta, bias=None) -> NormedDelta:
        """``delta`` (a tensor or ``SplitParts``; ``bias`` a vector added to every row first) as
        what this norm makes of it, for ``ResidualStream.push``."""
        if not self.has_bias:
            raise RuntimeError("a layer norm behind a sublayer has a weight and a bias")
        return NormedDelta(delta, self, None if bias is None else bias.float().contiguous())

    def forward(self, stream: ResidualStream, rows=None, n_rows: int = 0):
        rt = self.runtime
        if self.has_bias:
            n, name = (stream.x.shape[0], "normed") if rows is None else (n_rows, "normed_rows")
            h = rt.buffer(name, (n, self.dim), rt.act_dtype)
            settle_normed(rt, stream, h, norm=self, rows=rows, n_rows=n_rows)
            return h
        more_rows, more_vec = stream.take_more()
        delta = stream.take_pending()
        if rows is None:
            h = rt.buffer("normed", (stream.x.shape[0], self.dim), rt.act_dtype)
        else:
            h = rt.buffer("normed_rows", (n_rows, self.dim), rt.act_dtype)
        rt.ops.add_layernorm(stream.x, delta, self.weight, self.eps, h, rows=rows, n_rows=n_rows,
                             more_rows=more_rows, more_vec=more_vec)
        return h


class MappedDelta:
    """A sublayer's output that still has to pass an element-wise norm (and a per-channel
    scale) before it joins the residual stream: ``(n(delta + bias)) * scale``.  A consumer
    that knows the kind (``DynamicTanhNorm.forward``) applies the map in the pass in which it
    adds the delta; any other consumer gets the mapped values through ``resolve()`` (one
    kernel of its own, float32)."""

    def __init__(self, delta, norm: "DynamicTanhNorm", scale=None, bias=None):
        self.delta, self.norm, self.scale, self.bias = delta, norm, scale, bias

    @property
    def shape(self):
        return self.delta.shape

    def post(self) -> tuple:
        return (self.norm.alpha, self.norm.weight, self.norm.bias, self.scale)

    def release(self) -> None:
        if hasattr(self.delta, "release"):
            self.delta.release()

    def resolve(self):
        rt = self.norm.runtime
        t, d = self.delta.shape
        out = rt.buffer("mapped_delta", (t, d), torch.float32)
        rt.ops.add_tanh_norm(None, self.delta, None, None, post=self.post(), bias=self.bias,
                             y_out=out)
        return out

    def float(self):
        return self.resolve()


class DynamicTanhNorm(Norm):
    """``tanh(alpha * x) * w + b`` with a learned scalar ``alpha`` and vectors ``w``, ``b``: no
    mean, no variance, nothing reduced over the row; float32 inside, one rounding.

    Tensors: the weight under ``tensor_name`` ("" = the part's own prefix), ``alpha`` and
    ``b`` beside it.  As a block's first norm of a sublayer it adds the stream's pending
    delta in the same pass (``forward``); behind a sublayer it does not run by itself:
    ``mapped(delta, scale)`` wraps the sublayer's output, and whoever adds that to the
    stream applies the map while it reads the rows anyway."""

    decode_capturable = prompt_capturable = True

    def __init__(self, dim: int, tensor_name: str = "weight"):
        self.dim, self.tensor_name = int(dim), tensor_name
        self.weight = self.bias = None
        self.alpha = 1.0

    def _name(self, suffix: str) -> str:
        return f"{self.tensor_name}.{suffix}" if self.tensor_name else suffix

    def tensor_specs(self) -> dict:
        return {self.tensor_name: TensorSpec((self.dim,), kind="vector", init="ones"),
                self._name("b"): TensorSpec((self.dim,), kind="vector", init="zeros"),
                self._name("alpha"): TensorSpec((), kind="vector", init="ones")}

    def bind(self, tensors: dict, runtime) -> None:
        self.runtime = runtime
        self.weight = tensors[self.tensor_name].contiguous()
        self.bias = tensors[self._name("b")].to(self.weight.dtype).contiguous()
        self.alpha = float(tensors[self._name("alpha")])     # read once, at load time
        runtime.ops.require_part("tanhnorm")

    def mapped(self, delta, scale=None, bias=None) -> MappedDelta:
        """``delta`` (a tensor or ``SplitParts``; ``bias`` a vector added to every row first)
        as what this norm, then ``scale``, make of it, for ``ResidualStream.push``."""
        return MappedDelta(delta, self, scale, bias)

    def forward(self, stream: ResidualStream, rows=None, n_rows: int = 0):
        rt = self.runtime
        more_rows, more_vec = stream.take_more()
        if more_rows is not None or more_vec is not None:
            rt.ops.require_part("layernorm")
            rt.ops.residual_add(stream.x, more_rows, more_vec)
        delta = stream.take_pending()
        post = bias = None
        if isinstance(delta, MappedDelta):
            post, bias, delta = delta.post(), delta.bias, delta.delta
        if rows is None:
            h = rt.buffer("normed", (stream.x.shape[0], self.dim), rt.act_dtype)
        else:
            h = rt.buffer("normed_rows", (n_rows, self.dim), rt.act_dtype)
        rt.ops.add_tanh_norm(stream.x, delta, (self.alpha, self.weight, self.bias), h, post=post,
                             bias=bias, rows=rows, n_rows=n_rows)
        return h
