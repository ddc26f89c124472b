"""Matrix memories with ONE decay per head and token, run as their recurrence: linear attention without a softmax.

Per head, with S [key channels, value channels] starting at zero and carried from token to token:

    S <- a_t S + b_t k_t v_t^T;    o_t = S^T q_t

``Retention``: a is a constant of the head, b = 1; q and k are rotated by the position, k is multiplied by
dim^-1/2; y = unit(o) * silu(Wg x), unit(o) each head over its root mean square.

``ExponentialGateMemory`` (the matrix memory of an extended LSTM): q = Wq x * dim^-1/2; per head an input gate
i = cap tanh((Wi x + bi) / cap) and a forget gate f = log sigmoid(cap tanh((Wf x + bf) / cap)), and a running maximum
m_t = max(f_t + m_(t-1), i_t) with m = 0 before the first token, so that a_t = exp(f_t + m_(t-1) - m_t) and
b_t = exp(i_t - m_t) never overflow.  The keys are summed by the same recurrence, n <- a n + b k, and
o_t = S^T q_t / (max(|n . q|, exp(-m_t)) + 1e-6); y = unit(o) * w * sigmoid(Wg x) with a weight per channel of all heads.
n is one more value channel of S, whose value is always one: n . q is then one more column of the read-out.

Both end with Wo.  q, k, v and the output gate (and, where the step only brings a few single tokens, the exponential
gates' two rows per head, which otherwise are a product with a float result of their own) are ONE merged product of x.
Everything after the products is float:

* requests that bring one token: one kernel from the projection's row to the gated output (``kernels.memory_step``);
* portions of prompts, bfloat16, key sizes 64 and 128: chunks of 64 tokens on tensor cores (``csrc/memory_chunks.cu``),
  then the normaliser, norm and gate;
* everything else: float rows and the plain form of the recurrence in ``csrc/delta_rule.cu``.
"""
from __future__ import annotations

import math

import torch

from .. import kernels
from ..errors import Unsupported
from .base import Mixer, StateNeed, TensorSpec
from .position import RotaryHalf

DENOMINATOR_EPS = 1e-6    # added to the normaliser of the exponentially gated memory
LEAST_LOG_DECAY = -80.0   # a decay below e^-80 keeps nothing that a float can tell from zero


def _pad8(n: int) -> int:
    return -(-n // 8) * 8


class ScalarDecayMemory(Mixer):
    """What the two share: the merged projection q | k | v | g and the recurrence."""
    kernel_groups = ("recurrent",)
    ones = 0   # value channels whose value is one (they sum the keys)

    def __init__(self, hidden: int, heads: int, key_dim: int, value_dim: int, norm_eps: float, names: dict):
        if key_dim > 256:
            raise Unsupported(f"key size {key_dim}: the recurrence kernel holds up to 256 key channels per column")
        self.hidden, self.H, self.dk, self.dv = int(hidden), int(heads), int(key_dim), int(value_dim)
        self.eps, self.names = float(norm_eps), dict(names)
        qk, vw = self.H * self.dk, self.H * self.dv
        self.oq, self.ok = 0, _pad8(qk)
        self.ov = self.ok + _pad8(qk)
        self.og = self.ov + _pad8(vw)
        self.in_width = self.og + _pad8(vw)        # q | k | v | g
        self.full_width = self.in_width            # ... and what a subclass puts after them
        self.rt = None

    def tensor_specs(self):
        n, D = self.names, self.hidden
        qk, vw = self.H * self.dk, self.H * self.dv
        return [TensorSpec(n["q"], (qk, D)), TensorSpec(n["k"], (qk, D)), TensorSpec(n["v"], (vw, D)),
                TensorSpec(n["g"], (vw, D)), TensorSpec(n["o"], (D, vw))]

    def _memory_need(self):
        return StateNeed((self.H, self.dv + self.ones, self.dk), torch.float32, "S")

    # rows of the merged projection beyond q, k, v and g: (offset, tensor)
    def _more_rows(self, fetch):
        return []

    def bind(self, rt, fetch):
        self.rt = rt
        n = self.names
        w = torch.zeros((self.full_width, self.hidden), dtype=rt.dtype, device=rt.device)
        for off, t in [(off, fetch(n[name])) for off, name in ((self.oq, "q"), (self.ok, "k"), (self.ov, "v"),
                                                               (self.og, "g"))] + self._more_rows(fetch):
            w[off:off + t.shape[0]] = t
        self.w_full, self.w_in, self.w_more = w, w[:self.in_width], w[self.in_width:]
        self.w_o = fetch(n["o"])

    # rotation and constant factors of the queries and keys: (inverse frequencies, dims, q factor, k factor)
    def _rotation(self):
        return None, 0, 1.0, 1.0

    # the gates of the portions' rows: a_t and b_t (b None: one), or their logarithms, and exp(-m_t) (None: no normaliser)
    def _gates(self, z, step, state, T, logs: bool):
        raise NotImplementedError

    # the same for single tokens, as ``kernels.memory_step`` takes it
    def _step_gates(self, z, state):
        raise NotImplementedError

    def forward(self, x, step, cache, state):
        rt = self.rt
        x = rt.rows(x)
        T = x.shape[0]
        H, dk, dv, dvo = self.H, self.dk, self.dv, self.dv + self.ones
        f32 = torch.float32
        # (layers of other sizes have buffers of their own: one that only long steps use must not grow once CUDA graphs
        # hold the pool's addresses)
        size = f":{H}:{dk}:{dvo}"
        single, many = step.n_single, step.n_entries - step.n_single
        z = None
        if self.full_width > self.in_width and (rt.dtype == f32 or (many == 0 and T <= kernels.FEWROWS_MAX_ROWS)):
            # a few single tokens: the product is a stream of the weights, and a float result costs nothing
            proj = rt.scratch.get("memory_proj_full" + size, (rt.max_tokens if rt.dtype == f32 else kernels.FEWROWS_MAX_ROWS,
                                                       self.full_width), f32)[:T]
            rt.linear(proj, x, self.w_full)
            z = proj[:, self.in_width:]
        else:
            proj = rt.scratch.get("memory_proj" + size, (rt.max_tokens, self.in_width), rt.dtype)[:T]
            rt.linear(proj, x, self.w_in)
            if self.full_width > self.in_width:
                z = rt.scratch.get("memory_gate_z" + size, (rt.max_tokens, self.full_width - self.in_width), f32)[:T]
                rt.linear(z, x, self.w_more)
        S = state["S"] if isinstance(state, dict) else state
        inv_freq, rot_dims, q_mult, k_mult = self._rotation()
        den_eps = DENOMINATOR_EPS if self.ones else 0.0
        y = rt.scratch.get("delta_y", (rt.max_tokens, H * dv), rt.dtype)[:T]
        if single > 0:
            kernels.memory_step(y, proj, (self.oq, self.ok, self.ov, self.og), self._step_gates(z, state), S, inv_freq,
                                rot_dims, step.positions, step.cu_q, step.state_slot, single, H, dk, dv, q_mult, k_mult,
                                self.eps, weight=self.norm_w, den_eps=den_eps, silu_gate=self.silu_gate,
                                ones=bool(self.ones))
        if many > 0:
            chunks = kernels.memory_chunks_fits(rt.dtype, dk, dv) and rot_dims % 4 == 0
            decay, put, floor = self._gates(z, step, state, T, chunks)
            o = rt.scratch.get("delta_o" + size, (rt.max_tokens, H, dvo), f32)[:T]
            if chunks:
                v = proj[:, self.ov:]
                if rot_dims or k_mult != 1.0:   # (float rows that are no longer bfloat16: as two bfloat16 each)
                    halves = [rt.scratch.get(f"memory_split{i}{size}", (rt.max_tokens, H * dk), rt.dtype)[:T] for i in range(4)]
                    q, k = halves[:2], halves[2:]
                    kernels.memory_rotate_split(proj, (self.oq, self.ok), inv_freq, rot_dims, step.positions, q, k, H, dk,
                                                1.0, k_mult)
                else:
                    q, k = (proj[:, self.oq:], None), (proj[:, self.ok:], None)
                kernels.memory_chunks(q, k, v, decay, put, S, o, step.cu_q, step.state_slot, single, many, H, dk, dv, q_mult)
            else:
                qn = rt.scratch.get("delta_q" + size, (rt.max_tokens, H, dk), f32)[:T]
                kn = rt.scratch.get("delta_k" + size, (rt.max_tokens, H, dk), f32)[:T]
                vv = rt.scratch.get("delta_v" + size, (rt.max_tokens, H, dvo), f32)[:T]
                kernels.memory_prepare(proj, (self.oq, self.ok, self.ov), inv_freq, rot_dims, step.positions, qn, kn, vv,
                                       H, dk, dv, q_mult, k_mult, ones=bool(self.ones))
                kernels.memory_recurrence(qn, kn, vv, decay, put, S, o, step.cu_q, step.state_slot, many, H, dk, dvo,
                                          entry0=single)
            kernels.memory_output(y[single:], o[single:], proj[single:, self.og:], H, dv, self.eps, weight=self.norm_w,
                                  floor=floor[single:] if floor is not None else None, den_eps=den_eps,
                                  silu_gate=self.silu_gate)
        out = rt.scratch.get(self.out_key, (rt.max_tokens, self.hidden), rt.dtype)[:T]
        return rt.linear(out, y, self.w_o)


class Retention(ScalarDecayMemory):
    silu_gate = True
    norm_w = None

    def __init__(self, hidden: int, heads: int, key_dim: int, value_dim: int, decay, norm_eps: float, names: dict,
                 rotation: RotaryHalf = None):
        """``decay``: the constant decay of each head.  ``rotation``: a ``RotaryHalf`` over the key size in the
        rotate-half layout, or None.  ``names``: tensor names under the keys q, k, v, g, o."""
        super().__init__(hidden, heads, key_dim, value_dim, norm_eps, names)
        self.decay = [float(d) for d in decay]
        if len(self.decay) != self.H or any(not 0.0 <= d <= 1.0 for d in self.decay):
            raise Unsupported(f"a decay in [0, 1] for each of the {self.H} heads is wanted, not {self.decay}")
        self.rotation = rotation
        if rotation is not None and (rotation.head_dim != self.dk or rotation.interleaved
                                     or rotation.amplitude() is not None):
            raise Unsupported("a rotation of the key size in the rotate-half layout without an amplitude")

    def state_need(self):
        return self._memory_need()

    def bind(self, rt, fetch):
        super().bind(rt, fetch)
        # the same decay for every token: rows that nobody writes again
        self.decays = torch.tensor(self.decay, dtype=torch.float32, device=rt.device)
        self.decay_rows = self.decays.repeat(rt.max_tokens, 1)
        logs = [max(math.log(d), LEAST_LOG_DECAY) if d > 0 else LEAST_LOG_DECAY for d in self.decay]
        self.log_rows = torch.tensor(logs, dtype=torch.float32, device=rt.device).repeat(rt.max_tokens, 1)
        self.inv_freq = None
        if self.rotation is not None:
            self.rotation.bind(rt, fetch)
            self.inv_freq = self.rotation.rotary_table()[:self.rotation.rotary_dim // 2].contiguous()

    def _rotation(self):
        return self.inv_freq, (self.rotation.rotary_dim if self.rotation is not None else 0), 1.0, self.dk ** -0.5

    def _gates(self, z, step, state, T, logs):
        return (self.log_rows if logs else self.decay_rows)[:T], None, None

    def _step_gates(self, z, state):
        return self.decays


class ExponentialGateMemory(ScalarDecayMemory):
    silu_gate = False
    ones = 1

    def __init__(self, hidden: int, heads: int, key_dim: int, value_dim: int, gate_cap: float, norm_eps: float, names: dict):
        """``names``: tensor names under the keys q, k, v, g, o, norm, i, i_bias, f, f_bias."""
        super().__init__(hidden, heads, key_dim, value_dim, norm_eps, names)
        if not gate_cap > 0:
            raise Unsupported("gate_cap must be > 0")
        self.cap = float(gate_cap)
        self.full_width = self.in_width + _pad8(2 * self.H)   # the input gates' rows, then the forget gates'

    def tensor_specs(self):
        n, D = self.names, self.hidden
        return super().tensor_specs() + [
            TensorSpec(n["norm"], (self.H * self.dv,), role="vector", init="one_plus_normal"),
            TensorSpec(n["i"], (self.H, D)), TensorSpec(n["i_bias"], (self.H,), role="vector"),
            TensorSpec(n["f"], (self.H, D)), TensorSpec(n["f_bias"], (self.H,), role="vector")]

    def state_need(self):
        return [self._memory_need(), StateNeed((self.H,), torch.float32, "m")]

    def _more_rows(self, fetch):
        return [(self.in_width, fetch(self.names["i"])), (self.in_width + self.H, fetch(self.names["f"]))]

    def bind(self, rt, fetch):
        super().bind(rt, fetch)
        n = self.names
        self.i_bias, self.f_bias = fetch(n["i_bias"]).float().contiguous(), fetch(n["f_bias"]).float().contiguous()
        self.norm_w = fetch(n["norm"]).float().contiguous()

    def _rotation(self):
        return None, 0, self.dk ** -0.5, 1.0

    def _gates(self, z, step, state, T, logs):
        rt, H = self.rt, self.H
        decay, put, floor = (rt.scratch.get(f"{key}:{H}", (rt.max_tokens, H), torch.float32)[:T]
                             for key in ("memory_decay", "memory_put", "memory_floor"))
        kernels.memory_gates(z, self.i_bias, self.f_bias, self.cap, state["m"], step.cu_q, step.state_slot, decay, put,
                             floor, step.n_entries - step.n_single, H, entry0=step.n_single, logs=logs)
        return decay, put, floor

    def _step_gates(self, z, state):
        return (z, 0, self.H, self.i_bias, self.f_bias, self.cap, state["m"])
