"""Duzizen, written out plainly: whole sequences, float64, no cache, no state carried between calls, nothing imported
from the package.  One function per mechanism; ``forward`` puts them together from the configuration's JSON form and
a dict of tensors by name.  It is the oracle of ``tests/test_duzizen.py``.

Notation: h [T, D] the rows of one sequence, positions 0 .. T-1, ``w`` a dict name -> float64 tensor, ``p`` the prefix
of a part's tensor names.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64
GLU_SLOPE = 1.702
DENOMINATOR_EPS = 1e-6      # added to the normaliser of the matrix memory


# ---- small pieces -------------------------------------------------------------------------------------------
def rms_unit(x, eps):
    """x over the root of (its mean square along the last axis, plus eps)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, weight, bias, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * weight + bias


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(x):
    return x * torch.sigmoid(x)


def log_sigmoid(x):
    return torch.clamp(x, max=0.0) - torch.log1p(torch.exp(-x.abs()))


def causal_conv(u, taps_w):
    """u [T, C], taps_w [C, taps]: y[t] = sum_j taps_w[:, j] * u[t - (taps - 1) + j], with u = 0 at negative times."""
    T, C = u.shape
    taps = taps_w.shape[1]
    pad = torch.cat([torch.zeros((taps - 1, C), dtype=u.dtype), u], 0)
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + pad[j:j + T] * taps_w[:, j]
    return y


# ---- embedding ----------------------------------------------------------------------------------------------
def embedding(cfg, w, tokens):
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    b = (cfg.get("embedding") or {}).get("bigram")
    if b is not None:
        n = int(b["buckets"])
        rows = [n]
        for prev, cur in zip(tokens[:-1], tokens[1:]):
            rows.append((int(prev) * int(b["mul_prev"]) + int(cur) * int(b["mul_cur"])) % n)
        x = x + w["bigram"][torch.tensor(rows)]
    return x


def token_side(cfg, w, i, x, tokens, eps):
    """What layer i adds to the stream x for the tokens themselves."""
    dim = int(cfg["token_side"]["dim"])
    p = f"l{i}.side."
    e = w["side.embed"][torch.as_tensor(tokens, dtype=torch.long)][:, i * dim:(i + 1) * dim]
    y = (gelu_tanh(x @ w[p + "gate"].T) * e) @ w[p + "proj"].T
    return rms_unit(y, eps) * w[p + "norm"]


# ---- rotations ----------------------------------------------------------------------------------------------
def rotary_frequencies(rot):
    """Inverse frequencies of the dims / 2 pairs; with ``scaling`` the long wavelengths are stretched by a factor and
    those between two bounds by a mix."""
    dims, base = int(rot["dims"]), float(rot["base"])
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        sc = rot.get("scaling")
        if sc is not None:
            factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
            wavelength = 2 * math.pi / f
            if wavelength > original / low:
                f = f / factor
            elif not wavelength < original / high:
                s = (original / wavelength - low) / (high - low)
                f = (1 - s) * f / factor + s * f
        out.append(f)
    return out


def rotate(x, rot, interleaved):
    """x [T, heads, d]: the first rot.dims coordinates of each head turned by position * frequency."""
    T, dims = x.shape[0], int(rot["dims"])
    ang = torch.arange(T, dtype=F64)[:, None] * torch.tensor(rotary_frequencies(rot), dtype=F64)[None, :]
    cos, sin = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    out = x.clone()
    if interleaved:
        a, b = slice(0, dims, 2), slice(1, dims, 2)
    else:
        a, b = slice(0, dims // 2), slice(dims // 2, dims)
    u, v = x[..., a], x[..., b]
    out[..., a] = u * cos - v * sin
    out[..., b] = v * cos + u * sin
    return out


# ---- mixers -------------------------------------------------------------------------------------------------
def visible(T, mask):
    """[T, T] bool: which key j (column) the query at i (row) sees."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if mask is not None:
        seen = seen & ((i - j < int(mask["size"])) | (j < int(mask.get("keep_first", 0))))
    return seen


def softmax_plus_one(s, seen):
    """exp(s_j) / (1 + sum exp(s_j)) over the keys seen."""
    s = s.masked_fill(~seen, float("-inf"))
    top = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def key_is_value_attention(m, w, p, h, eps):
    T = h.shape[0]
    H, G, d = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q, k = h @ w[p + "q"].T, h @ w[p + "k"].T
    if int(m.get("conv") or 0) > 0:
        q, k = causal_conv(q, w[p + "q.conv"]), causal_conv(k, w[p + "k.conv"])
    v = k.reshape(T, G, d)
    q = (rms_unit(q, eps) * w[p + "q.norm"]).reshape(T, H, d)
    k = (rms_unit(k, eps) * w[p + "k.norm"]).reshape(T, G, d)
    if m.get("rot") is not None:
        q, k = rotate(q, m["rot"], True), rotate(k, m["rot"], True)
    kv_of = [hd // (H // G) for hd in range(H)]
    s = torch.einsum("ihd,jhd->hij", q, k[:, kv_of]) * float(m["scale"])
    a = softmax_plus_one(s, visible(T, m.get("mask"))[None])
    o = torch.einsum("hij,jhd->ihd", a, v[:, kv_of])
    return o.reshape(T, H * d) @ w[p + "o"].T


def retention(m, w, p, h, eps):
    T = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ w[p + "q"].T).reshape(T, H, d)
    k = (h @ w[p + "k"].T).reshape(T, H, d)
    v = (h @ w[p + "v"].T).reshape(T, H, dv)
    if m.get("rot") is not None:
        q, k = rotate(q, m["rot"], False), rotate(k, m["rot"], False)
    k = k * d ** -0.5
    decay = torch.tensor([float(x) for x in m["decay"]], dtype=F64)[:, None, None]
    S = torch.zeros((H, d, dv), dtype=F64)
    o = torch.zeros((T, H, dv), dtype=F64)
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S, q[t])
    o = rms_unit(o, eps).reshape(T, H * dv) * silu(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def parallel(m, w, p, h, eps):
    a = key_is_value_attention(m["left"], w, p + "left.", h, eps)
    b = retention(m["right"], w, p + "right.", h, eps)
    return 0.5 * (rms_unit(a, eps) * w[p + "left.out"] + rms_unit(b, eps) * w[p + "right.out"])


def matrix_memory(m, w, p, h, eps):
    T = h.shape[0]
    H, d, dv, cap = int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"])
    q = (h @ w[p + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).reshape(T, H, d)
    v = (h @ w[p + "v"].T).reshape(T, H, dv)
    gi = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    gf = log_sigmoid(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    S, n, top = torch.zeros((H, d, dv), dtype=F64), torch.zeros((H, d), dtype=F64), torch.zeros(H, dtype=F64)
    o = torch.zeros((T, H, dv), dtype=F64)
    for t in range(T):
        new = torch.maximum(gf[t] + top, gi[t])
        keep, put = torch.exp(gf[t] + top - new)[:, None], torch.exp(gi[t] - new)[:, None]
        top = new
        S = keep[:, :, None] * S + put[:, :, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep * n + put * k[t]
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-top)) + DENOMINATOR_EPS
        o[t] = torch.einsum("hkv,hk->hv", S, q[t]) / den[:, None]
    o = rms_unit(o, eps).reshape(T, H * dv) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


# ---- feed-forwards ------------------------------------------------------------------------------------------
def dense_ffn(w, p, h):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(w, p, h, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(GLU_SLOPE * g) * (u + 1)) @ w[p + "down"].T


def experts(m, w, p, h):
    s = torch.sigmoid(h @ w[p + "router"].T)
    n, top, limit = int(m["router"]["experts"]), int(m["router"]["top"]), float(m["expert"]["limit"])
    chosen = torch.topk(s, top, dim=-1).indices
    out = torch.zeros_like(h)
    for e in range(n):
        rows = (chosen == e).any(-1).nonzero().reshape(-1)
        if rows.numel():
            out[rows] += expert(w, p + f"e{e}.", s[rows, e][:, None] * h[rows], limit)
    return out


def feed_forward(m, w, p, h):
    return experts(m, w, p, h) if m["kind"] == "moe" else dense_ffn(w, p, h)


# ---- the model ----------------------------------------------------------------------------------------------
def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence.  ``layers_out``: a list that gets the stream after every layer."""
    w = {k: v.to(F64) if v.is_floating_point() else v for k, v in w.items()}
    eps = float(cfg["norm"]["eps"])
    tokens = [int(t) for t in tokens]

    def norm(name, x):
        return layer_norm(x, w[name], w[name + ".b"], eps)

    x = embedding(cfg, w, tokens)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mixer = {"mlstm": matrix_memory, "parallel": parallel}[layer["type"]]
        x = x + norm(p + "norm1b", mixer(layer["mixer"], w, p + "mix.", norm(p + "norm1", x), eps))
        if layer.get("mlp") is not None:
            x = x + norm(p + "norm2b", feed_forward(layer["mlp"], w, p + "mlp.", norm(p + "norm2", x)))
        if cfg.get("token_side") is not None:
            x = x + token_side(cfg, w, i, x, tokens, eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm("final.norm", x) @ w["head"].T


def generate(cfg, w, prompt, n):
    """Greedy continuation (ties -> lowest id)."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(torch.argmax(forward(cfg, w, toks)[-1]).item()))
    return toks[len(prompt):]


greedy = generate
