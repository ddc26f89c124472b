"""Toripel, written out plainly: whole sequences, float64, no cache, no state carried, nothing imported from
the package.  One function per mechanism; ``forward`` puts them together from the configuration's JSON form
and a dict of tensors by name.  It is the oracle of ``tests/test_toripel.py``.

Notation: T tokens of one sequence at positions 0 .. T-1, x [T, S, D] the S copies of the residual stream, ``w`` a
dict name -> float64 tensor (tables of integers as they are).
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64
UNIT_EPS = 1e-6


def rms_unit(x, eps):
    """x over the root of (its mean square along the last axis, plus eps)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30.0))))


def causal_conv(u, taps_w):
    """u [T, C], taps_w [C, taps]: y[t] = sum_j taps_w[:, j] * u[t - (taps - 1) + j], with u = 0 at negative times."""
    T, C = u.shape
    taps = taps_w.shape[1]
    pad = torch.cat([torch.zeros((taps - 1, C), dtype=u.dtype), u], 0)
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + pad[j:j + T] * taps_w[:, j]
    return y


# ---- the stream and its copies -------------------------------------------------------------------------------
def embedding(cfg, w, tokens):
    return w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * float(cfg["embedding"]["scale"])


def read_streams(x, weights):
    """One sublayer's input: the copies added up with a weight each."""
    return (x * weights[None, :, None]).sum(1)


def write_streams(x, y, mix, out):
    """The copies after a sublayer: every new one a mix of all old ones plus its share of the output."""
    new = [sum(mix[a, b] * x[:, a] for a in range(x.shape[1])) + out[b] * y for b in range(x.shape[1])]
    return torch.stack(new, 1)


def norm(cfg, w, name, u):
    return rms_unit(u, float(cfg["norm"]["eps"])) * (1.0 + w[name])


# ---- rotation --------------------------------------------------------------------------------------------------
def rotary_frequencies(rot):
    """Inverse frequencies of the dims / 2 pairs and the factor on cos and sin (1 without scaling)."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if sc is None:
        return f, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def where(turns):
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(where(float(sc["fast"]))), 0)
    hi = min(math.ceil(where(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x, rot):
    """x [T, heads, d]: the pairs (2 i, 2 i + 1) of the first rot.dims coordinates turned by position * frequency."""
    dims = int(rot["dims"])
    f, m = rotary_frequencies(rot)
    ang = torch.arange(x.shape[0], dtype=F64)[:, None] * torch.tensor(f, dtype=F64)[None, :]
    cos, sin = (torch.cos(ang) * m)[:, None, :], (torch.sin(ang) * m)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def visible(T, mask):
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    seen = j <= i
    if mask is not None:
        seen = seen & (i - j < int(mask["size"]))
    return seen


# ---- mixers ------------------------------------------------------------------------------------------------------
def attention(m, w, p, h, eps):
    """Grouped-query attention over a window, no positions: biases, unit-size heads of q and k, a plain softmax."""
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms_unit((h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, d), eps)
    k = rms_unit((h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, d), eps)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, dv)
    group = [hd // (H // G) for hd in range(H)]
    s = torch.einsum("ihd,jhd->hij", q, k[:, group]) * float(m["scale"])
    a = torch.softmax(s.masked_fill(~visible(T, m.get("mask"))[None], float("-inf")), -1)
    return torch.einsum("hij,jhd->ihd", a, v[:, group]).reshape(T, H * dv) @ w[p + "o"].T


def latent_rows(m, w, p, h, eps):
    """What a latent attention layer leaves per token: c [T, rank] and the rotated shared key part [T, rot_dim]."""
    R = int(m["kv_rank"])
    both = h @ w[p + "dkv"].T
    c = rms_unit(both[:, :R], eps) * w[p + "dkv.norm"]
    return c, rotate(both[:, None, R:], m["rot"])[:, 0]


def latent_attention(m, w, p, h, eps, rows):
    T = h.shape[0]
    H, d, r, dv = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"])
    c, kr = rows
    cq = rms_unit(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).reshape(T, H, d + r)
    qn, qr = q[..., :d], rotate(q[..., d:], m["rot"])
    kn = (c @ w[p + "uk"].T).reshape(T, H, d)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    s = (torch.einsum("ihd,jhd->hij", qn, kn) + torch.einsum("ihd,jd->hij", qr, kr)) * float(m["scale"])
    s = s.masked_fill(~visible(T, m.get("mask"))[None], float("-inf"))
    sink = w[p + "sink"][:, None, None].expand(H, T, 1)
    a = torch.softmax(torch.cat([s, sink], -1), -1)[..., :T]      # the sink has no value
    return torch.einsum("hij,jhd->ihd", a, v).reshape(T, H * dv) @ w[p + "o"].T


def gated_delta(m, w, p, h, eps):
    """The delta rule with one decay per head, read after the token's own write."""
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = silu(causal_conv(h @ w[p + "q"].T, w[p + "q.conv"])).reshape(T, G, d)
    k = silu(causal_conv(h @ w[p + "k"].T, w[p + "k.conv"])).reshape(T, G, d)
    v = silu(causal_conv(h @ w[p + "v"].T, w[p + "v.conv"])).reshape(T, H, dv)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + UNIT_EPS) * d ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + UNIT_EPS)
    beta = torch.sigmoid(h @ w[p + "b"].T)                                                    # [T, H]
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))   # [T, H]
    group = [hd // (H // G) for hd in range(H)]
    q, k = q[:, group], k[:, group]
    S = torch.zeros((H, d, dv), dtype=F64)
    o = torch.zeros((T, H, dv), dtype=F64)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    o = rms_unit(o, eps) * w[p + "norm"]
    return (o.reshape(T, H * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- feed-forward --------------------------------------------------------------------------------------------------
def table_experts(m, w, p, h, tokens):
    """Experts that a table names for every token id, each with the same weight."""
    top = int(m["router"]["top"])
    chosen = w[p + "table"][torch.as_tensor(tokens, dtype=torch.long)].long()      # [T, top]
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in chosen[t].tolist():
            q = f"{p}e{e}."
            y[t] += (silu(w[q + "gate"] @ h[t]) * (w[q + "up"] @ h[t])) @ w[q + "down"].T / top
    return y


# ---- the model -----------------------------------------------------------------------------------------------------
def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence.  ``layers_out``: a list that gets the sum of the copies after every layer."""
    w = {k: v.to(F64) if v.is_floating_point() else v for k, v in w.items()}
    eps = float(cfg["norm"]["eps"])
    tokens = [int(t) for t in tokens]
    e = embedding(cfg, w, tokens)
    x = torch.stack([e] * int(cfg["streams"]), 1)
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m, t = f"l{i}.", layer["mixer"], layer["type"]
        h = norm(cfg, w, p + "norm1", read_streams(x, w[p + "hc1.in"]))
        if t == "attention":
            y = attention(m, w, p + "mix.", h, eps)
        elif t == "delta":
            y = gated_delta(m, w, p + "mix.", h, eps)
        elif t == "latent_attention":
            if m.get("kv_from") is not None:
                rows = kept[int(m["kv_from"])]
            else:
                rows = kept[i] = latent_rows(m, w, p + "mix.", h, eps)
            y = latent_attention(m, w, p + "mix.", h, eps, rows)
        else:
            raise ValueError(f"layer type {t!r}")
        x = write_streams(x, y, w[p + "hc1.mix"], w[p + "hc1.out"])
        if layer.get("mlp") is not None:
            h = norm(cfg, w, p + "norm2", read_streams(x, w[p + "hc2.in"]))
            y = table_experts(layer["mlp"], w, p + "mlp.", h, tokens)
            x = write_streams(x, y, w[p + "hc2.mix"], w[p + "hc2.out"])
        if layers_out is not None:
            layers_out.append(x.sum(1))
    return norm(cfg, w, "final.norm", x.sum(1)) @ w["head"].T
