"""Typed configuration of Duzizen, a decoder whose config.json lists its layers one by one.

    {"architecture": "Duzizen", "vocab": V, "width": D, "norm": {"eps": e},
     "embedding": {"bigram": {"buckets": n, "mul_prev": a, "mul_cur": b}},      (bigram optional)
     "token_side": {"dim": d},                                                  (optional)
     "layers": [{"type": T, "mixer": {...}, "mlp": {...} | null}, ...]}

Mixer types and their keys:

* ``mlstm``: heads, dim, vdim, gate_cap.
* ``parallel``: two mixers on the same input, ``left`` {heads, kv_heads, dim, vdim (= dim: the values are the keys),
  scale, ``conv`` (taps; optional), ``mask`` {size, ``keep_first``} (optional), ``rot`` {dims, base, ``scaling`` {factor,
  low, high, original}} (both optional)} and ``right`` {heads, dim, vdim, decay [heads], ``rot`` {dims, base}
  (optional)}.

Feed-forwards: {"kind": "dense", "ff": F} or {"kind": "moe", "expert": {"ff": F, "limit": l}, "router": {"experts": E,
"top": k}}.  Nothing here is a default for a size: a missing key is an error.
"""
from __future__ import annotations

import dataclasses
from typing import Optional, Tuple

from ..errors import ModelConfigInvalid
from .tugelorn import _get

ARCHITECTURE = "Duzizen"
MEMORY_TYPE = "mlstm"
PARALLEL_TYPE = "parallel"


@dataclasses.dataclass(frozen=True)
class WavelengthScaling:
    factor: float
    low: float
    high: float
    original: float


@dataclasses.dataclass(frozen=True)
class Rotation:
    dims: int
    base: float
    scaling: Optional[WavelengthScaling] = None


@dataclasses.dataclass(frozen=True)
class MemoryConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float
    type: str = MEMORY_TYPE


@dataclasses.dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    conv: int = 0                     # taps; 0: no convolution
    window: Optional[int] = None
    keep_first: int = 0
    rot: Optional[Rotation] = None


@dataclasses.dataclass(frozen=True)
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot: Optional[Rotation] = None


@dataclasses.dataclass(frozen=True)
class ParallelConfig:
    left: AttentionConfig
    right: RetentionConfig
    type: str = PARALLEL_TYPE


@dataclasses.dataclass(frozen=True)
class DenseConfig:
    ff: int
    kind: str = "dense"


@dataclasses.dataclass(frozen=True)
class ExpertsConfig:
    experts: int
    top: int
    expert_ff: int
    limit: float
    kind: str = "moe"


@dataclasses.dataclass(frozen=True)
class LayerConfig:
    mixer: object
    mlp: object      # DenseConfig, ExpertsConfig or None

    @property
    def type(self) -> str:
        return self.mixer.type


@dataclasses.dataclass(frozen=True)
class PairTable:
    buckets: int
    mul_prev: int
    mul_cur: int


def _bad(text: str):
    raise ModelConfigInvalid("config.json: " + text)


def _positive(where: str, **values) -> None:
    for name, v in values.items():
        if not v > 0:
            _bad(f"{where}.{name} must be > 0")


def _count(j, key: str, where: str) -> int:
    """A whole number that may be 0."""
    v = j.get(key) if isinstance(j, dict) else None
    if isinstance(v, bool) or not isinstance(v, int) or not 0 <= v < 2 ** 31:
        _bad(f"{where}.{key} must be a whole number >= 0, got {v!r}")
    return v


def _rotation(j, where: str, dim: int) -> Optional[Rotation]:
    if j.get("rot") is None:
        return None
    rj, where = j["rot"], where + ".rot"
    scaling = None
    if isinstance(rj, dict) and rj.get("scaling") is not None:
        sw = where + ".scaling"
        scaling = WavelengthScaling(*(_get(rj["scaling"], k, sw, float) for k in ("factor", "low", "high", "original")))
        _positive(sw, factor=scaling.factor, low=scaling.low, original=scaling.original)
        if scaling.high < scaling.low:
            _bad(f"{sw}: low must not exceed high")
    rot = Rotation(_get(rj, "dims", where, int), _get(rj, "base", where, float), scaling)
    if rot.dims <= 0 or rot.dims % 2 or rot.dims > dim or rot.base <= 0:
        _bad(f"{where}: dims must be even and lie in 2 .. dim, base > 0")
    return rot


def _rotation_json(rot: Rotation) -> dict:
    j = {"dims": rot.dims, "base": rot.base}
    if rot.scaling is not None:
        j["scaling"] = dataclasses.asdict(rot.scaling)
    return j


def _attention(j, where: str) -> AttentionConfig:
    heads, kv, dim, vdim = (_get(j, k, where, int) for k in ("heads", "kv_heads", "dim", "vdim"))
    _positive(where, heads=heads, kv_heads=kv, dim=dim)
    if heads % kv:
        _bad(f"{where}: heads must be a multiple of kv_heads")
    if vdim != dim:
        _bad(f"{where}: the values are the keys, so vdim must equal dim")
    window, keep = None, 0
    if j.get("mask") is not None:
        window = _get(j["mask"], "size", where + ".mask", int)
        if j["mask"].get("keep_first") is not None:
            keep = _count(j["mask"], "keep_first", where + ".mask")
    conv = _count(j, "conv", where) if j.get("conv") is not None else 0
    return AttentionConfig(heads, kv, dim, _get(j, "scale", where, float), conv, window, keep, _rotation(j, where, dim))


def _retention(j, where: str) -> RetentionConfig:
    heads, dim, vdim = (_get(j, k, where, int) for k in ("heads", "dim", "vdim"))
    _positive(where, heads=heads, dim=dim, vdim=vdim)
    decay = j.get("decay")
    if (not isinstance(decay, list) or len(decay) != heads
            or any(isinstance(d, bool) or not isinstance(d, (int, float)) or not 0 <= d <= 1 for d in decay)):
        _bad(f"{where}.decay must list a number in [0, 1] for each of the {heads} heads")
    return RetentionConfig(heads, dim, vdim, tuple(float(d) for d in decay), _rotation(j, where, dim))


def _mlp(j, where: str):
    if j is None:
        return None
    kind = j.get("kind") if isinstance(j, dict) else None
    if kind == "dense":
        q = DenseConfig(_get(j, "ff", where, int))
        _positive(where, ff=q.ff)
        return q
    if kind == "moe":
        ej, rj = j.get("expert"), j.get("router")
        q = ExpertsConfig(_get(rj, "experts", where + ".router", int), _get(rj, "top", where + ".router", int),
                          _get(ej, "ff", where + ".expert", int), _get(ej, "limit", where + ".expert", float))
        _positive(where, experts=q.experts, top=q.top, ff=q.expert_ff, limit=q.limit)
        if q.top > q.experts:
            _bad(f"{where}.router: top must not exceed experts")
        return q
    _bad(f"{where}.kind {kind!r} is neither 'dense' nor 'moe'")


@dataclasses.dataclass(frozen=True)
class DuzizenConfig:
    vocab: int
    width: int
    layers: Tuple[LayerConfig, ...]
    norm_eps: float
    pair: Optional[PairTable] = None
    side_dim: Optional[int] = None
    architecture: str = ARCHITECTURE

    @property
    def vocab_size(self) -> int:
        return self.vocab

    # -- json --------------------------------------------------------------
    @classmethod
    def from_json(cls, j: dict) -> "DuzizenConfig":
        vocab, width = _get(j, "vocab", "top", int), _get(j, "width", "top", int)
        eps = _get(j.get("norm"), "eps", "norm", float)
        _positive("top", vocab=vocab, width=width, eps=eps)
        pair = None
        ej = j.get("embedding")
        if isinstance(ej, dict) and ej.get("bigram") is not None:
            bw = "embedding.bigram"
            pair = PairTable(_get(ej["bigram"], "buckets", bw, int), _count(ej["bigram"], "mul_prev", bw),
                             _count(ej["bigram"], "mul_cur", bw))
        side = None
        if j.get("token_side") is not None:
            side = _get(j["token_side"], "dim", "token_side", int)
            _positive("token_side", dim=side)
        raw = j.get("layers")
        if not isinstance(raw, list) or not raw:
            _bad("'layers' must be a list with at least one layer")
        layers = []
        for i, lj in enumerate(raw):
            where = f"layers[{i}]"
            if not isinstance(lj, dict) or "type" not in lj or not isinstance(lj.get("mixer"), dict) or "mlp" not in lj:
                _bad(f"{where} needs 'type', 'mixer' and 'mlp' (null for none)")
            mj, mw = lj["mixer"], where + ".mixer"
            if lj["type"] == MEMORY_TYPE:
                mixer = MemoryConfig(*(_get(mj, k, mw, int) for k in ("heads", "dim", "vdim")),
                                     _get(mj, "gate_cap", mw, float))
                _positive(mw, heads=mixer.heads, dim=mixer.dim, vdim=mixer.vdim, gate_cap=mixer.gate_cap)
            elif lj["type"] == PARALLEL_TYPE:
                if not isinstance(mj.get("left"), dict) or not isinstance(mj.get("right"), dict):
                    _bad(f"{mw} needs 'left' and 'right'")
                mixer = ParallelConfig(_attention(mj["left"], mw + ".left"), _retention(mj["right"], mw + ".right"))
            else:
                _bad(f"{where}.type {lj['type']!r} is not one of {(MEMORY_TYPE, PARALLEL_TYPE)}")
            layers.append(LayerConfig(mixer, _mlp(lj["mlp"], where + ".mlp")))
        return cls(vocab, width, tuple(layers), eps, pair, side)

    def to_json(self) -> dict:
        layers = []
        for layer in self.layers:
            m, q = layer.mixer, layer.mlp
            if m.type == MEMORY_TYPE:
                mj = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap}
            else:
                a, r = m.left, m.right
                lj = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.dim, "scale": a.scale}
                if a.conv:
                    lj["conv"] = a.conv
                if a.window is not None:
                    lj["mask"] = {"size": a.window, "keep_first": a.keep_first}
                rj = {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "decay": list(r.decay)}
                for side, half in ((lj, a), (rj, r)):
                    if half.rot is not None:
                        side["rot"] = _rotation_json(half.rot)
                mj = {"left": lj, "right": rj}
            pj = None
            if q is not None and q.kind == "dense":
                pj = {"kind": "dense", "ff": q.ff}
            elif q is not None:
                pj = {"kind": "moe", "expert": {"ff": q.expert_ff, "limit": q.limit},
                      "router": {"experts": q.experts, "top": q.top}}
            layers.append({"type": m.type, "mixer": mj, "mlp": pj})
        j = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
             "norm": {"eps": self.norm_eps}, "layers": layers}
        if self.pair is not None:
            j["embedding"] = {"bigram": dataclasses.asdict(self.pair)}
        if self.side_dim is not None:
            j["token_side"] = {"dim": self.side_dim}
        return j
