"""A residual stream kept as several copies (hyper-connections).

Instead of one stream there are S, all equal to the embedding's rows at the start.  A sublayer reads a weighted sum of
them and writes to all of them at once:

    u = sum_s in[s] x_s;   y = sublayer(norm(u));   x_t <- sum_s mix[s, t] x_s + out[t] y       (mix is [from, to])

and the model's last norm reads their plain sum.  ``StreamsNorm`` is the norm of such a weighted sum and
``StreamsConnection`` the weights with which an output enters; ``HyperConnectionBlock`` arranges them around a mixer and a
feed-forward.  As in the other pre-norm blocks a sublayer's output is left pending and the norm that follows makes the
sum: one kernel mixes the copies, adds the output (or the rows of a mixture's experts, which it adds up itself) and norms
what the next sublayer reads.  While all copies are equal there is one of them.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import kernels
from ..errors import Unsupported
from .base import Block, ExpertRows, FeedForward, Mixer, Norm, Part, Residual, TensorSpec


def _check_streams(n: int) -> int:
    if not (1 <= int(n) <= kernels.MAX_STREAMS):
        raise Unsupported(f"{n} copies of the stream: 1 to {kernels.MAX_STREAMS}")
    return int(n)


class StreamsNorm(Norm):
    """y = u / rms(u) * (weight_offset + w), u the sum of the copies, each times its weight of the tensor ``in_name`` (None:
    the plain sum)."""

    def __init__(self, dim: int, streams: int, eps: float, weight_name: str, in_name: Optional[str] = None,
                 weight_offset: float = 0.0, scratch_key: str = "normed"):
        self.dim, self.streams, self.eps = int(dim), _check_streams(streams), float(eps)
        self.weight_name, self.in_name, self.weight_offset = weight_name, in_name, float(weight_offset)
        self.scratch_key = scratch_key
        self.weight = self.weights_in = None
        self.rt = None

    def tensor_specs(self):
        specs = [TensorSpec(self.weight_name, (self.dim,), role="vector",
                            init="normal" if self.weight_offset else "one_plus_normal")]
        if self.in_name is not None:
            specs.append(TensorSpec(self.in_name, (self.streams,), role="vector", init="one_plus_normal"))
        return specs

    def bind(self, rt, fetch):
        self.rt = rt
        self.weight = (fetch(self.weight_name).float() + self.weight_offset).contiguous()
        self.weights_in = fetch(self.in_name).float().contiguous() if self.in_name is not None else None

    def from_table(self, h, table, scale: float, ids, pending):
        """The embedding's rows h = table[ids] * scale and this norm of S copies of them, in one kernel."""
        rt = self.rt
        if table.dtype != rt.dtype or table.shape[1] != self.dim or not table.is_contiguous():
            return None
        y = rt.scratch.get(self.scratch_key, (rt.max_tokens, self.dim), rt.dtype)[:h.shape[0]]
        kernels.streams_step(y, None, self.streams, self.weight, self.eps, self.weights_in, x_out=h, table=table, ids=ids,
                             scale=scale, pending=pending, status=rt.status)
        return y

    def fold(self, stream: Residual, rows=None, n_rows=None):
        rt = self.rt
        T = stream.h.shape[0]
        ready, stream.ready = stream.ready, None
        if ready is not None and rows is None and ready[0] is self and stream.pending is None:
            return ready[1]
        x = stream.copies if stream.copies is not None else stream.h
        args = {}
        if stream.pending is not None:
            args = {"mix": stream.connection.mix, "weights_out": stream.connection.out}
            if isinstance(stream.pending, ExpertRows):
                args["pairs"] = stream.pending.args
            else:
                args["delta"] = rt.rows(stream.pending)
        if rows is None:
            y = rt.scratch.get(self.scratch_key, (rt.max_tokens, self.dim), rt.dtype)[:T]
            if args:
                if stream.copies is None:
                    stream.copies = rt.scratch.get("stream_copies", (rt.max_tokens, self.streams, self.dim),
                                                   torch.float32)[:T]
                args["x_out"] = stream.copies
            kernels.streams_step(y, x, self.streams, self.weight, self.eps, self.weights_in, status=rt.status, **args)
            stream.pending = stream.connection = None   # it is part of the copies now
        else:
            n = rows.numel() if n_rows is None else n_rows
            y = rt.scratch.get(self.scratch_key + "_rows", (rt.max_tokens, self.dim), rt.dtype)[:n]
            kernels.streams_step(y, x, self.streams, self.weight, self.eps, self.weights_in, row_idx=rows, n_rows=n,
                                 status=rt.status, **args)
        return y

    def apply(self, x):
        y = torch.empty_like(x)   # one stream, outside a step
        kernels.rmsnorm(y, x, self.weight, self.eps)
        return y


class StreamsConnection(Part):
    """The weights with which a sublayer's output enters the copies: ``mix`` [from, to] and ``out``."""

    def __init__(self, streams: int, names: dict):
        """``names``: tensor names under the keys mix, out."""
        self.streams, self.names = _check_streams(streams), dict(names)
        self.mix = self.out = None

    def tensor_specs(self):
        S = self.streams
        return [TensorSpec(self.names["mix"], (S, S), role="vector", init="eye_plus_normal"),
                TensorSpec(self.names["out"], (S,), role="vector", init="one_plus_normal")]

    def bind(self, rt, fetch):
        self.mix = fetch(self.names["mix"]).float().contiguous()
        self.out = fetch(self.names["out"]).float().contiguous()


class HyperConnectionBlock(Block):
    """x_t <- sum_s mix1[s, t] x_s + out1[t] Mixer(norm1(x)); then the same with the feed-forward (which, with its norm and
    connection, may be absent).  The norms are ``StreamsNorm``."""

    def __init__(self, norm1: StreamsNorm, mixer: Mixer, connect1: StreamsConnection, norm2: Optional[StreamsNorm] = None,
                 ffn: Optional[FeedForward] = None, connect2: Optional[StreamsConnection] = None):
        if (ffn is None) != (norm2 is None) or (ffn is None) != (connect2 is None):
            raise ValueError("a feed-forward comes with its norm and its connection, or none of the three is given")
        self.norm1, self.mixer, self.connect1 = norm1, mixer, connect1
        self.norm2, self.ffn, self.connect2 = norm2, ffn, connect2

    def _parts(self):
        return [p for p in (self.norm1, self.mixer, self.connect1, self.norm2, self.ffn, self.connect2) if p is not None]

    @property
    def graph_safe(self):
        return all(p.graph_safe for p in self._parts())

    @property
    def kernel_groups(self):
        return tuple(dict.fromkeys(g for p in self._parts() for g in getattr(p, "kernel_groups", ())))

    def tensor_specs(self):
        return [s for p in self._parts() for s in p.tensor_specs()]

    def bind(self, rt, fetch):
        for p in self._parts():
            p.bind(rt, fetch)

    @property
    def first_norm(self):
        return self.norm1

    def forward(self, stream: Residual, step, cache, state) -> None:
        stream.takes_unscaled = False
        step.residual_sink = None
        x = self.norm1.fold(stream)
        stream.pending = self.mixer.forward(x, step, cache, state)
        stream.connection = self.connect1
        if self.ffn is not None:
            x = self.norm2.fold(stream)
            step.takes_expert_rows = True      # (the sum that follows adds a token's expert rows up itself)
            stream.pending = self.ffn.forward(x, step)
            step.takes_expert_rows = False
            stream.connection = self.connect2
