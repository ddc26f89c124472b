"""Duzizen put together from the parts: exponentially gated matrix memories, and pairs of an attention and a retention on
the same input.

A layer is a ``SandwichNormBlock`` of layer norms with a token side input last: h += norm1b(mixer(norm1(h)));
h += norm2b(ff(norm2(h))); h += side(h, token).  The mixers: ``ExponentialGateMemory``; ``ParallelMixers`` of a
``GroupedQueryAttention`` whose values are its keys (short convolutions on q and k, norms over the whole projections,
interleaved pairs of part of a head rotated with stretched long wavelengths, a window beside which the first tokens
stay visible, a sink of score zero) and a ``Retention``, half the sum of the two normed outputs.  The feed-forward is
``GeluGLU`` or a ``MixtureOfExperts`` with sigmoid scores, not renormalised, that multiply the experts' input.  The
embedding is the token's row plus a row of a second table chosen by the pair (previous token, token).

Tensor names: ``embed``, ``bigram``, ``side.embed``, ``l<i>.norm1 / norm1b / norm2 / norm2b`` each with a ``.b``,
``l<i>.mix.*`` (``.left.*`` and ``.right.*`` in a pair), ``l<i>.mlp.gate / up / down`` or ``l<i>.mlp.router`` and
``l<i>.mlp.e<k>.gate / up / down``, ``l<i>.side.gate / proj / norm``, ``final.norm`` and ``final.norm.b``, ``head``.
"""
from __future__ import annotations

from .. import kernels
from ..config.duzizen import MEMORY_TYPE, DenseConfig, DuzizenConfig
from ..engine.plan import ModelPlan, RunEntry
from ..parts import (ExponentialGateMemory, GeluGLU, GroupedQueryAttention, LayerNorm, MixtureOfExperts, NoPosition,
                     OutputHead, ParallelMixers, Retention, RotaryHalf, SandwichNormBlock, TokenEmbedding, TokenSideInput)

PAIR_SHARE = 0.5         # each half's share of a pair's output
SINK_SCORE = 0.0         # one is added to every softmax denominator
GLU_SLOPE = 1.702        # an expert's gate is g * sigmoid(1.702 g) ...
GLU_UP_SHIFT = 1.0       # ... times (u + 1)


def _memory(cfg: DuzizenConfig, m, p: str):
    names = {"q": p + "q", "k": p + "k", "v": p + "v", "g": p + "g", "o": p + "o", "norm": p + "norm", "i": p + "i",
             "i_bias": p + "i.b", "f": p + "f", "f_bias": p + "f.b"}
    return ExponentialGateMemory(cfg.width, m.heads, m.dim, m.vdim, m.gate_cap, cfg.norm_eps, names)


def _attention(cfg: DuzizenConfig, m, p: str):
    hd = GroupedQueryAttention.kernel_head_dim(m.dim, m.dim)
    position = NoPosition()
    if m.rot is not None:
        sc = m.rot.scaling
        stretched = None if sc is None else {"factor": sc.factor, "low": sc.low, "high": sc.high, "original": sc.original}
        # (without a scaling: the frequencies evaluated in float64 and rounded once)
        position = RotaryHalf(hd, m.rot.base, rotary_dim=m.rot.dims, interleaved=True, wavelength_scaling=stretched,
                              linear_scaling=1.0 if stretched is None else None)
    names = {"q": p + "q", "k": p + "k", "o": p + "o", "q_norm": p + "q.norm", "k_norm": p + "k.norm"}
    if m.conv:
        names.update({"q_conv": p + "q.conv", "k_conv": p + "k.conv"})
    return GroupedQueryAttention(cfg.width, m.heads, m.kv_heads, m.dim, position, names, qk_norm_eps=cfg.norm_eps,
                                 window=m.window, scale=m.scale, value_dim=m.dim, conv_taps=m.conv,
                                 keep_first=m.keep_first, sink_score=SINK_SCORE, keys_as_values=True)


def _retention(cfg: DuzizenConfig, m, p: str):
    rotation = None
    if m.rot is not None:
        sc = m.rot.scaling
        stretched = None if sc is None else {"factor": sc.factor, "low": sc.low, "high": sc.high, "original": sc.original}
        rotation = RotaryHalf(m.dim, m.rot.base, rotary_dim=m.rot.dims, wavelength_scaling=stretched,
                              linear_scaling=1.0 if stretched is None else None)
    names = {"q": p + "q", "k": p + "k", "v": p + "v", "g": p + "g", "o": p + "o"}
    return Retention(cfg.width, m.heads, m.dim, m.vdim, m.decay, cfg.norm_eps, names, rotation)


def _mixer(cfg: DuzizenConfig, m, p: str):
    if m.type == MEMORY_TYPE:
        return _memory(cfg, m, p)
    return ParallelMixers(cfg.width, _attention(cfg, m.left, p + "left."), _retention(cfg, m.right, p + "right."),
                          PAIR_SHARE, PAIR_SHARE, out_norms=(p + "left.out", p + "right.out", cfg.norm_eps))


def _feed_forward(cfg: DuzizenConfig, q, p: str):
    if isinstance(q, DenseConfig):
        return GeluGLU(cfg.width, q.ff, {"gate": p + "gate", "up": p + "up", "down": p + "down"})
    names = {"router": p + "router", "gate": p + "e{e}.gate", "up": p + "e{e}.up", "down": p + "e{e}.down"}
    return MixtureOfExperts(cfg.width, q.experts, q.top, q.expert_ff, names,
                            activation=kernels.GluAct.clamped(q.limit, GLU_SLOPE, GLU_UP_SHIFT),
                            rule=kernels.RouteRule("sigmoid"), weight_on_input=True)


def build_plan(cfg: DuzizenConfig) -> ModelPlan:
    D, eps = cfg.width, cfg.norm_eps
    n_layers = len(cfg.layers)

    def norm(name):
        return LayerNorm(D, eps, name, name + ".b")

    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        norm2 = ffn = post2 = side = None
        if layer.mlp is not None:
            norm2, post2 = norm(p + "norm2"), norm(p + "norm2b")
            ffn = _feed_forward(cfg, layer.mlp, p + "mlp.")
        if cfg.side_dim is not None:
            side = TokenSideInput(cfg.vocab, D, cfg.side_dim, i * cfg.side_dim, n_layers * cfg.side_dim, eps,
                                  {"table": "side.embed", "gate": p + "side.gate", "proj": p + "side.proj",
                                   "norm": p + "side.norm"})
        layers.append(SandwichNormBlock(norm(p + "norm1"), _mixer(cfg, layer.mixer, p + "mix."), norm(p + "norm1b"), norm2,
                                        ffn, post2, side=side))
    pair = None
    if cfg.pair is not None:
        pair = {"name": "bigram", "buckets": cfg.pair.buckets, "mul_prev": cfg.pair.mul_prev, "mul_cur": cfg.pair.mul_cur}
    return ModelPlan(embedding=TokenEmbedding(cfg.vocab, D, "embed", pair=pair), layers=layers,
                     order=[RunEntry(i) for i in range(n_layers)], final_norm=norm("final.norm"),
                     head=OutputHead(D, cfg.vocab, "head"), vocab_size=cfg.vocab, max_position=None)
