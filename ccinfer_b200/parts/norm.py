"""Norms.  RMSNorm: y = x * rsqrt(mean(x^2) + eps) * w (7QiC/ccInfer: src/kernel/norm/rms_norm.cu:24-60)."""
from __future__ import annotations

import torch

from .. import kernels
from .base import Norm, Residual, TensorSpec, UnscaledRows


class RMSNorm(Norm):
    def __init__(self, dim: int, eps: float, weight_name: str, scratch_key: str = "normed", weight_offset: float = 0.0,
                 weight_scale: float = 1.0, scalar: bool = False):
        """``scalar``: the stored weight is ONE number for all coordinates (a tensor of no axes); it is spread over
        the ``dim`` places of the kernels' weight vector when it is bound.
        ``weight_offset`` c: the stored weight lies around zero and the norm multiplies by (c + w); the sum is
        made once, in float, when the weight is bound (exact for a bfloat16 w of ordinary size).
        ``weight_scale`` s: the norm's rows times s (a constant factor on what a product makes of them, a
        model's scale on its logits for instance, costs nothing here)."""
        self.weight_scale = float(weight_scale)
        self.dim, self.eps, self.weight_name, self.scratch_key = int(dim), float(eps), weight_name, scratch_key
        self.weight_offset = float(weight_offset)
        self.scalar = bool(scalar)
        self.w = None
        self.rt = None

    def tensor_specs(self):
        return [TensorSpec(self.weight_name, () if self.scalar else (self.dim,), role="vector",
                           init="normal" if self.weight_offset else "one_plus_normal")]

    def bind(self, rt, fetch):
        self.rt = rt
        self.w = fetch(self.weight_name)
        if self.scalar:
            self.w = self.w.float().reshape(1).expand(self.dim).contiguous()
        if self.weight_offset:
            self.w = (self.w.float() + self.weight_offset).contiguous()
        if self.weight_scale != 1.0:
            self.w = (self.w.float() * self.weight_scale).contiguous()

    def spec(self):
        """This norm as ``kernels.norm_chain`` takes it."""
        return kernels.NormSpec("rms", self.w, None, self.eps)

    def fold(self, stream: Residual, rows=None, n_rows=None):
        rt = self.rt
        T = stream.h.shape[0]
        ready, stream.ready = stream.ready, None
        if ready is not None and rows is None and ready[0] is self and stream.pending is None:
            return ready[1]   # written together with the stream (the embedding's kernel)
        un, stream.unscaled = stream.unscaled, None
        if un is not None and rows is None and un.norm is self and stream.pending is None:
            # the product before did the sum and left this norm's rows short of their factor
            return un if stream.takes_unscaled else un.finish()
        # (rows left for another norm than this one: h is complete, they are dropped)
        if rows is None:
            y = rt.scratch.get(self.scratch_key, (rt.max_tokens, self.dim), rt.dtype)[:T]
            kernels.residual_rmsnorm(y, stream.h, stream.pending, self.w, self.eps, status=rt.status)
            stream.pending = None  # it is part of h now
        else:
            n = rows.numel() if n_rows is None else n_rows
            y = rt.scratch.get(self.scratch_key + "_rows", (rt.max_tokens, self.dim), rt.dtype)[:n]
            kernels.residual_rmsnorm(y, stream.h, stream.pending, self.w, self.eps, row_idx=rows, n_rows=n,
                                     status=rt.status)
        return y

    def from_embedding(self, h, table, ids, pending):
        """norm(h) for h = table[ids], both written by one kernel; None where that kernel does not apply."""
        rt = self.rt
        if table.dtype != rt.dtype or table.shape[1] != self.dim or not table.is_contiguous():
            return None
        y = rt.scratch.get(self.scratch_key, (rt.max_tokens, self.dim), rt.dtype)[:h.shape[0]]
        kernels.embed_rmsnorm(y, h, table, ids, self.w, self.eps, status=rt.status, pending=pending)
        return y

    def unscaled_rows_from(self, stream: Residual, xw, ssq, parts: int):
        """What a product that adds into the stream itself leaves for this norm: ``xw`` gets h * w, ``ssq``
        [16, parts] the partial sums of h^2 (see ``Runtime.linear``).  None: this norm takes no such rows."""
        if xw.shape[1] != self.dim:
            return None
        h = stream.h
        return UnscaledRows(xw, ssq, parts, self.dim, self.eps, self, lambda: self.rows_of(h))

    def rows_of(self, h):
        """norm(h) of a stream that is complete (nothing pending), as a plain tensor."""
        rt = self.rt
        y = rt.scratch.get(self.scratch_key, (rt.max_tokens, self.dim), rt.dtype)[:h.shape[0]]
        kernels.residual_rmsnorm(y, h, None, self.w, self.eps, status=rt.status)
        return y

    def apply(self, x):
        y = torch.empty_like(x)  # the part alone, outside a step: not a buffer of the pool
        kernels.rmsnorm(y, x, self.w, self.eps)
        return y


class LayerNorm(Norm):
    """y = (x - mean) / sqrt(mean((x - mean)^2) + eps) * weight + bias, over the stream's float rows
    (``kernels.norm_chain``).  (Its weights are not called ``w``: a part that looks for an RMS norm's weight to fold
    into a kernel of its own does not find one here.)"""

    def __init__(self, dim: int, eps: float, weight_name: str, bias_name: str, scratch_key: str = "normed"):
        self.dim, self.eps, self.scratch_key = int(dim), float(eps), scratch_key
        self.weight_name, self.bias_name = weight_name, bias_name
        self.weight = self.bias = None
        self.rt = None

    def tensor_specs(self):
        return [TensorSpec(self.weight_name, (self.dim,), role="vector", init="one_plus_normal"),
                TensorSpec(self.bias_name, (self.dim,), role="vector")]

    def bind(self, rt, fetch):
        self.rt = rt
        self.weight = fetch(self.weight_name).float().contiguous()
        self.bias = fetch(self.bias_name).float().contiguous()

    def spec(self):
        return kernels.NormSpec("layer", self.weight, self.bias, self.eps)

    def fold(self, stream: Residual, rows=None, n_rows=None):
        rt = self.rt
        T = stream.h.shape[0]
        ready, stream.ready = stream.ready, None
        stream.unscaled = None
        if ready is not None and rows is None and ready[0] is self and stream.pending is None:
            return ready[1]
        delta = None if stream.pending is None else rt.rows(stream.pending)
        if rows is None:
            y = rt.scratch.get(self.scratch_key, (rt.max_tokens, self.dim), rt.dtype)[:T]
            kernels.norm_chain(stream.h, delta, nxt=self.spec(), y=y, status=rt.status)
            stream.pending = None
        else:
            n = rows.numel() if n_rows is None else n_rows
            y = rt.scratch.get(self.scratch_key + "_rows", (rt.max_tokens, self.dim), rt.dtype)[:n]
            kernels.norm_chain(stream.h, delta, nxt=self.spec(), y=y, row_idx=rows, n_rows=n, status=rt.status)
        return y

    def apply(self, x):
        y = torch.empty_like(x)
        kernels.norm_chain(x.float().contiguous(), nxt=self.spec(), y=y, status=self.rt.status)
        return y


class StreamRows(Norm):
    """No norm at all: the rows of the stream itself, in the compute type, for a sublayer that reads the stream as it
    is.  A block that starts with such a sublayer names one of these as its ``first_norm``, so that whoever writes
    the stream last (the embedding, the block before) can leave the rows ready in the same pass.  In the 32-bit
    path the rows ARE the stream."""

    def __init__(self, dim: int, scratch_key: str = "stream_rows"):
        self.dim, self.scratch_key = int(dim), scratch_key
        self.rt = None
        self._ones = None

    def bind(self, rt, fetch):
        self.rt = rt

    def buffer(self, T: int):
        rt = self.rt
        return rt.scratch.get(self.scratch_key, (rt.max_tokens, self.dim), rt.dtype)[:T]

    def fold(self, stream: Residual, rows=None, n_rows=None):
        rt = self.rt
        if rows is not None:
            raise NotImplementedError("the stream's own rows are not gathered by index")
        ready, stream.ready = stream.ready, None
        stream.unscaled = None
        pending, stream.pending = stream.pending, None
        if pending is None:
            if rt.dtype == torch.float32:
                return stream.h
            if ready is not None and isinstance(ready[0], StreamRows):
                return ready[1]
        y = None if rt.dtype == torch.float32 else self.buffer(stream.h.shape[0])
        if pending is not None:   # a sum that the part before left to whoever reads the stream next
            if self._ones is None:
                self._ones = torch.ones(self.dim, dtype=torch.float32, device=rt.device)
            kernels.scaled_residual(stream.h, rt.rows(pending), self._ones, y=y)
        else:
            kernels.postnorm_residual(stream.h, None, None, 0.0, 0.0, y=y)
        return stream.h if y is None else y

    def apply(self, x):
        return x
