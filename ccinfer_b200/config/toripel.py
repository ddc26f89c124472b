"""Typed configuration of Toripel, a decoder whose config.json lists its layers one by one.

    {"architecture": "Toripel", "vocab": V, "width": D, "streams": S, "norm": {"eps": e}, "embedding": {"scale": s},
     "layers": [{"type": T, "mixer": {...}, "mlp": {"kind": "moe", "expert": {"ff": F},
                                                    "router": {"experts": E, "top": n}} | null}, ...]}

Mixer types and their keys:

* ``attention``: heads, kv_heads, dim, vdim, scale, ``mask`` {size}.
* ``latent_attention``: heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, ``rot`` {dims, base,
  ``scaling`` {factor, original, fast, slow}}, ``mask`` {size}, and optionally ``kv_from``: the layer whose cached rows
  this one reads instead of making its own.
* ``delta``: heads, kv_heads, dim, vdim, conv (taps).

``mask`` and ``rot.scaling`` are taken where they are present (without a mask every earlier token is seen).  Nothing
here is a default for a size: a missing key is an error.
"""
from __future__ import annotations

import dataclasses
from typing import Optional, Tuple

from ..errors import ModelConfigInvalid
from .gevovik import Rotation, _rotation, _rotation_json
from .tugelorn import _get

ARCHITECTURE = "Toripel"
ATTENTION_TYPE = "attention"
LATENT_TYPE = "latent_attention"
DELTA_TYPE = "delta"


@dataclasses.dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int] = None
    type: str = ATTENTION_TYPE


@dataclasses.dataclass(frozen=True)
class LatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot: Rotation
    window: Optional[int] = None
    kv_from: Optional[int] = None
    type: str = LATENT_TYPE


@dataclasses.dataclass(frozen=True)
class DeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    type: str = DELTA_TYPE


@dataclasses.dataclass(frozen=True)
class MoeConfig:
    experts: int
    top: int
    expert_ff: int
    kind: str = "moe"


@dataclasses.dataclass(frozen=True)
class LayerConfig:
    mixer: object
    mlp: Optional[MoeConfig]

    @property
    def type(self) -> str:
        return self.mixer.type


def _sizes(j, keys, where):
    return [_get(j, k, where, int) for k in keys]


def _window(mj, where) -> Optional[int]:
    if mj.get("mask") is None:
        return None
    return _sizes(mj["mask"], ("size",), where + ".mask")[0]


def _attention(mj, where) -> AttentionConfig:
    m = AttentionConfig(*_sizes(mj, ("heads", "kv_heads", "dim", "vdim"), where), _get(mj, "scale", where, float),
                        _window(mj, where))
    if m.heads % m.kv_heads:
        raise ModelConfigInvalid(f"config.json: {where}: heads must be a multiple of kv_heads")
    return m


def _latent(mj, where, i, layers) -> LatentConfig:
    heads, dim, rot_dim, vdim, kv_rank, q_rank = _sizes(mj, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"), where)
    kv_from = mj.get("kv_from")
    if kv_from is not None and (isinstance(kv_from, bool) or not isinstance(kv_from, int) or not (0 <= kv_from < i)):
        raise ModelConfigInvalid(f"config.json: {where}.kv_from must name an earlier layer")
    m = LatentConfig(heads, dim, rot_dim, vdim, kv_rank, q_rank, _get(mj, "scale", where, float),
                     _rotation(mj.get("rot") or {}, where + ".rot", rot_dim, "rot_dim"), _window(mj, where), kv_from)
    if kv_from is not None:
        src = layers[kv_from].mixer
        if (src.type != LATENT_TYPE or src.kv_from is not None or src.kv_rank != m.kv_rank or src.rot_dim != m.rot_dim
                or src.rot != m.rot):
            raise ModelConfigInvalid(f"config.json: {where}.kv_from: layer {kv_from} must be a latent attention layer with "
                                     f"rows of its own and the same kv_rank, rot_dim and rot")
    return m


def _delta(mj, where) -> DeltaConfig:
    m = DeltaConfig(*_sizes(mj, ("heads", "kv_heads", "dim", "vdim", "conv"), where))
    if m.heads % m.kv_heads:
        raise ModelConfigInvalid(f"config.json: {where}: heads must be a multiple of kv_heads")
    return m


def _mlp(pj, where) -> Optional[MoeConfig]:
    if pj is None:
        return None
    if not isinstance(pj, dict) or pj.get("kind") != "moe":
        raise ModelConfigInvalid(f"config.json: {where}.kind must be 'moe'")
    experts, top = _sizes(pj.get("router"), ("experts", "top"), where + ".router")
    if top > experts:
        raise ModelConfigInvalid(f"config.json: {where}.router: top is at most experts")
    return MoeConfig(experts, top, _sizes(pj.get("expert"), ("ff",), where + ".expert")[0])


@dataclasses.dataclass(frozen=True)
class ToripelConfig:
    vocab: int
    width: int
    streams: int
    layers: Tuple[LayerConfig, ...]
    norm_eps: float
    embed_scale: float
    architecture: str = ARCHITECTURE

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_json(cls, j: dict) -> "ToripelConfig":
        vocab, width, streams = _sizes(j, ("vocab", "width", "streams"), "top")
        eps = _get(j.get("norm"), "eps", "norm", float)
        if eps <= 0:
            raise ModelConfigInvalid("config.json: norm.eps must be > 0")
        scale = _get(j.get("embedding"), "scale", "embedding", float)
        raw = j.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ModelConfigInvalid("config.json: 'layers' must be a list with at least one layer")
        layers = []
        for i, lj in enumerate(raw):
            where = f"layers[{i}]"
            if (not isinstance(lj, dict) or "type" not in lj or not isinstance(lj.get("mixer"), dict) or "mlp" not in lj):
                raise ModelConfigInvalid(f"config.json: {where} needs 'type', 'mixer' and 'mlp' (null for none)")
            t, mj, mw = lj["type"], lj["mixer"], where + ".mixer"
            if t == ATTENTION_TYPE:
                mixer = _attention(mj, mw)
            elif t == LATENT_TYPE:
                mixer = _latent(mj, mw, i, layers)
            elif t == DELTA_TYPE:
                mixer = _delta(mj, mw)
            else:
                raise ModelConfigInvalid(f"config.json: {where}.type {t!r} is not one of "
                                         f"{(ATTENTION_TYPE, LATENT_TYPE, DELTA_TYPE)}")
            layers.append(LayerConfig(mixer, _mlp(lj["mlp"], where + ".mlp")))
        return cls(vocab, width, streams, tuple(layers), eps, scale)

    def to_json(self) -> dict:
        layers = []
        for layer in self.layers:
            m = layer.mixer
            if m.type == ATTENTION_TYPE:
                mj = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
            elif m.type == LATENT_TYPE:
                mj = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank,
                      "q_rank": m.q_rank, "scale": m.scale, "rot": _rotation_json(m.rot)}
                if m.kv_from is not None:
                    mj["kv_from"] = m.kv_from
            else:
                mj = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv}
            if getattr(m, "window", None) is not None:
                mj["mask"] = {"size": m.window}
            q = layer.mlp
            mlp = None if q is None else {"kind": q.kind, "expert": {"ff": q.expert_ff},
                                          "router": {"experts": q.experts, "top": q.top}}
            layers.append({"type": m.type, "mixer": mj, "mlp": mlp})
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "streams": self.streams,
                "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embed_scale}, "layers": layers}
