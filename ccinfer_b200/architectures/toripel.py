"""Toripel put together from the parts: a stream of several copies, windowed attention without positions, latent
attention whose queries are low-rank too and whose layers may read an earlier one's cached rows, a gated delta rule with
one decay per head, and experts that a table names for every token id.

A layer is a ``HyperConnectionBlock`` of ``StreamsNorm`` norms whose stored weights lie around zero (the factor is
1 + w).  The mixers: ``GroupedQueryAttention`` with biases and norms without weights on the q and k heads;
``LatentAttention`` over a window with a sink, rotated in interleaved pairs whose slow ones may be stretched, optionally
without rows of its own (``RunEntry.cache_of``); ``HeadGatedDelta``.  The feed-forward is a ``MixtureOfExperts`` of gated
experts with a table in place of a router.

Tensor names: ``embed``, ``l<i>.norm1 / norm2``, ``l<i>.hc1.in / mix / out`` and ``l<i>.hc2.*``, ``l<i>.mix.*``,
``l<i>.mlp.table`` and ``l<i>.mlp.e<k>.gate / up / down``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.toripel import ATTENTION_TYPE, LATENT_TYPE, ToripelConfig
from ..engine.plan import ModelPlan, RunEntry
from ..parts import (GroupedQueryAttention, HeadGatedDelta, HyperConnectionBlock, LatentAttention, MixtureOfExperts,
                     NoPosition, OutputHead, StreamsConnection, StreamsNorm, TokenEmbedding)

NORM_WEIGHT_OFFSET = 1.0   # the model's norms multiply by (1 + w)


def _attention(cfg: ToripelConfig, m, p: str):
    names = {k: p + k for k in ("q", "k", "v", "o")}
    names.update({"q_bias": p + "q.b", "k_bias": p + "k.b", "v_bias": p + "v.b"})
    return GroupedQueryAttention(cfg.width, m.heads, m.kv_heads, m.dim, NoPosition(), names, qk_norm_eps=cfg.norm_eps,
                                 window=m.window, scale=m.scale, value_dim=m.vdim, qk_norm_weights=False,
                                 tensor_core_heads=True)


def _latent(cfg: ToripelConfig, m, p: str):
    names = {"dq": p + "dq", "dq_norm": p + "dq.norm", "uq": p + "uq", "dkv": p + "dkv", "dkv_norm": p + "dkv.norm",
             "uk": p + "uk", "uv": p + "uv", "sink": p + "sink", "o": p + "o"}
    sc = m.rot.scaling
    ramp = None if sc is None else {"factor": sc.factor, "original": sc.original, "fast": sc.fast, "slow": sc.slow}
    return LatentAttention(cfg.width, m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.window, m.scale, m.rot.base,
                           m.rot.dims, cfg.norm_eps, names, interleaved=True, own_kv=m.kv_from is None,
                           q_rank=m.q_rank, ramp_scaling=ramp)


def _delta(cfg: ToripelConfig, m, p: str):
    names = {k: p + k for k in ("q", "k", "v", "o", "g", "a", "b", "A_log", "dt_bias", "norm")}
    names.update({"q_conv": p + "q.conv", "k_conv": p + "k.conv", "v_conv": p + "v.conv"})
    return HeadGatedDelta(cfg.width, m.heads, m.kv_heads, m.dim, m.vdim, m.conv, cfg.norm_eps, names)


def _mixer(cfg: ToripelConfig, m, p: str):
    if m.type == ATTENTION_TYPE:
        return _attention(cfg, m, p)
    return _latent(cfg, m, p) if m.type == LATENT_TYPE else _delta(cfg, m, p)


def build_plan(cfg: ToripelConfig) -> ModelPlan:
    D, S, eps = cfg.width, cfg.streams, cfg.norm_eps

    def norm(name, connection=None):
        return StreamsNorm(D, S, eps, name, in_name=connection and connection + ".in", weight_offset=NORM_WEIGHT_OFFSET)

    def connect(name):
        return StreamsConnection(S, {"mix": name + ".mix", "out": name + ".out"})

    layers, order = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        feed = ()
        if layer.mlp is not None:
            q = layer.mlp
            names = {"table": p + "mlp.table", "gate": p + "mlp.e{e}.gate", "up": p + "mlp.e{e}.up",
                     "down": p + "mlp.e{e}.down"}
            feed = (norm(p + "norm2", p + "hc2"),
                    MixtureOfExperts(D, q.experts, q.top, q.expert_ff, names, activation="swiglu", table_vocab=cfg.vocab),
                    connect(p + "hc2"))
        layers.append(HyperConnectionBlock(norm(p + "norm1", p + "hc1"), _mixer(cfg, layer.mixer, p + "mix."),
                                           connect(p + "hc1"), *feed))
        # (no layer runs twice: a layer's number is its place in the order)
        order.append(RunEntry(i, cache_of=getattr(layer.mixer, "kv_from", None)))
    return ModelPlan(embedding=TokenEmbedding(cfg.vocab, D, "embed", scale=cfg.embed_scale), layers=layers, order=order,
                     final_norm=norm("final.norm"), head=OutputHead(D, cfg.vocab, "head"), vocab_size=cfg.vocab,
                     max_position=None)
