"""A pair of mixers on the same rows, their results added with a constant factor each,

    out = left_scale * left(h) + right_scale * right(h),

or each result first over its root mean square, times a weight per channel (``out_norms``):

    out = left_scale * unit(left(h)) * w_left + right_scale * unit(right(h)) * w_right.

What the pair keeps is what its halves keep: the cache of the one that has one (at most one of them may), and the
states of both (the step hands each half its own).
"""
from __future__ import annotations

import torch

from .. import kernels
from ..errors import Unsupported
from .base import Mixer, NormedPair, TensorSpec


class ParallelMixers(Mixer):
    def __init__(self, hidden: int, left: Mixer, right: Mixer, left_scale: float, right_scale: float,
                 out_norms: tuple = None):
        """``out_norms``: (tensor of w_left, tensor of w_right, eps)."""
        if left.cache_need() is not None and right.cache_need() is not None:
            raise Unsupported("a pair of mixers on the same rows: at most one of them keeps a paged cache")
        self.hidden, self.left, self.right = int(hidden), left, right
        self.left_scale, self.right_scale = float(left_scale), float(right_scale)
        # each half leaves its result in a buffer of its own
        self.left.out_key, self.right.out_key = "mix_left_out", "mix_right_out"
        self.out_norms = tuple(out_norms) if out_norms is not None else None
        self.rt = None

    @property
    def graph_safe(self):
        return self.left.graph_safe and self.right.graph_safe

    @property
    def kernel_groups(self):
        return tuple(self.left.kernel_groups) + tuple(self.right.kernel_groups)

    @property
    def own_kv(self):
        return getattr(self.left, "own_kv", False) or getattr(self.right, "own_kv", False)

    def tensor_specs(self):
        own = [TensorSpec(name, (self.hidden,), role="vector", init="one_plus_normal")
               for name in (self.out_norms[:2] if self.out_norms is not None else ())]
        return self.left.tensor_specs() + self.right.tensor_specs() + own

    def cache_need(self):
        return self.left.cache_need() or self.right.cache_need()

    @staticmethod
    def _needs(mixer, side):
        sn = mixer.state_need()
        if sn is None:
            return []
        sn = list(sn) if isinstance(sn, (list, tuple)) else [sn]
        import dataclasses
        return [dataclasses.replace(n, name=f"{side}.{n.name}") for n in sn]

    def state_need(self):
        needs = self._needs(self.left, "left") + self._needs(self.right, "right")
        return needs or None

    def bind(self, rt, fetch):
        self.rt = rt
        self.left.bind(rt, fetch)
        self.right.bind(rt, fetch)
        if self.out_norms is not None:
            self.w_left, self.w_right = (fetch(n).float().contiguous() for n in self.out_norms[:2])

    @staticmethod
    def _state_of(mixer, side, state):
        sn = mixer.state_need()
        if sn is None:
            return None
        if isinstance(sn, (list, tuple)):
            return {n.name: state[f"{side}.{n.name}"] for n in sn}
        return state[f"{side}.{sn.name}"]

    def forward(self, x, step, cache, state):
        rt = self.rt
        x = rt.rows(x)
        T = x.shape[0]
        lc = cache if self.left.cache_need() is not None else None
        rc = cache if self.right.cache_need() is not None else None
        a = self.left.forward(x, step, lc, self._state_of(self.left, "left", state))
        b = self.right.forward(x, step, rc, self._state_of(self.right, "right", state))
        if self.out_norms is not None:   # the block's own sum makes it
            return NormedPair(rt.rows(a), rt.rows(b), self.w_left, self.w_right, self.left_scale, self.right_scale,
                              self.out_norms[2], self._finish)
        out = rt.scratch.get(self.out_key, (rt.max_tokens, self.hidden), rt.dtype)[:T]
        kernels.scaled_sum(out, rt.rows(a), rt.rows(b), self.left_scale, self.right_scale)
        return out

    def _finish(self, pair: NormedPair):
        rt = self.rt
        T = pair.a.shape[0]
        total = rt.scratch.get("mix_pair_sum", (rt.max_tokens, self.hidden), torch.float32)[:T].zero_()
        out = rt.scratch.get(self.out_key, (rt.max_tokens, self.hidden), rt.dtype)[:T]
        kernels.norm_chain(total, pair.a, y=out, pair=pair.args, status=rt.status)
        return out
