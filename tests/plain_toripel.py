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


def generate(cfg, w, prompt, n):
    """Greedy continuation (ties -> lowest id)."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(torch.argmax(forward(cfg, w, toks)[-1]).item()))
    return toks[len(prompt):]


greedy = generate


# ---- configurations of the tests and random weights ------------------------------------------------------------------
def attend(heads, kv_heads, dim, vdim, scale, window=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    return ("attention", m)


def latent(heads, dim, rot_dim, vdim, rank, q_rank, scale, window=None, base=10000.0, scaling=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "scale": scale,
         "rot": {"dims": rot_dim, "base": base}}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if window is not None:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return ("latent_attention", m)


def delta(heads, kv_heads, dim, vdim, conv):
    return ("delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv})


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def model(vocab, width, streams, eps, layers, scale=1.0):
    """``layers``: [((type, mixer), feed-forward or None)]."""
    return {"architecture": "Toripel", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
            "embedding": {"scale": scale}, "layers": [{"type": t, "mixer": m, "mlp": q} for (t, m), q in layers]}


# name -> (configuration, page size)
CONFIGS = {
    # windows of 24, 40 and 9 over the same latent rows (pages of 8), 17 in the attention layer; a layer without a
    # feed-forward; two copies of the stream
    "A": (model(96, 64, 2, 1e-5, [
        (latent(3, 8, 4, 12, 16, 20, 0.3, window=24, scaling=(4.0, 64, 8.0, 1.0)), moe(5, 2, 24)),
        (delta(4, 2, 8, 16, 4), moe(6, 3, 16)),
        (latent(2, 12, 4, 8, 16, 8, 0.35, window=40, scaling=(4.0, 64, 8.0, 1.0), kv_from=0), None),
        (attend(4, 2, 16, 24, 0.4, window=17), moe(4, 1, 32)),
        (latent(4, 8, 4, 16, 16, 24, 0.3, window=9, scaling=(4.0, 64, 8.0, 1.0), kv_from=0), moe(5, 2, 24))],
        scale=3.0), 8),
    # sizes that are multiples of nothing, one head, one copy of the stream, no masks, no scaling, one tap, every expert
    # used
    "B": (model(70, 44, 1, 1e-6, [
        (attend(1, 1, 10, 6, 0.5), moe(3, 3, 11)),
        (latent(1, 6, 2, 10, 12, 7, 0.4, base=500.0), moe(2, 1, 20)),
        (delta(1, 1, 6, 10, 1), None),
        (latent(2, 5, 2, 3, 12, 9, 0.6, base=500.0, kv_from=1), moe(7, 2, 9))]), 4),
    # what the tensor-core kernels take, heads laid out in a larger size among them; more copies than there are kernels
    # of a fixed number for
    "C": (model(128, 96, 5, 1e-5, [
        (latent(4, 16, 16, 16, 32, 48, 0.25, window=36, base=1000.0), moe(8, 2, 48)),
        (attend(8, 2, 72, 88, 0.15, window=33), moe(8, 4, 32)),
        (delta(4, 2, 64, 32, 2), moe(8, 2, 48)),
        (attend(4, 4, 40, 64, 0.2, window=70), None),
        (latent(6, 32, 16, 24, 32, 64, 0.2, window=100, base=1000.0, kv_from=0), moe(16, 1, 64)),
        (delta(3, 3, 128, 64, 3), moe(4, 2, 64))], scale=2.0), 16),
    # a window of one token, keys of more than 128 channels, four copies
    "D": (model(64, 128, 4, 1e-5, [
        (delta(2, 1, 160, 24, 4), moe(9, 2, 40)),
        (attend(2, 1, 64, 32, 0.3, window=1), None),
        (latent(2, 16, 16, 32, 48, 32, 0.3, window=1), moe(3, 1, 24)),
        (attend(6, 2, 128, 128, 0.12, window=20), moe(9, 2, 40))], scale=0.7), 16),
}


def config(name):
    return CONFIGS[name]


def tensor_shapes(cfg):
    D, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    s = {"embed": (V, D), "final.norm": (D,), "head": (V, D)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, t = f"l{i}.", layer["mixer"], layer["type"]
        q = p + "mix."
        H = m["heads"]
        if t == "attention":
            G, d, dv = m["kv_heads"], m["dim"], m["vdim"]
            s.update({q + "q": (H * d, D), q + "q.b": (H * d,), q + "k": (G * d, D), q + "k.b": (G * d,),
                      q + "v": (G * dv, D), q + "v.b": (G * dv,), q + "o": (D, H * dv)})
        elif t == "delta":
            qk, vw = m["kv_heads"] * m["dim"], H * m["vdim"]
            s.update({q + "q": (qk, D), q + "q.conv": (qk, m["conv"]), q + "k": (qk, D), q + "k.conv": (qk, m["conv"]),
                      q + "v": (vw, D), q + "v.conv": (vw, m["conv"]), q + "b": (H, D), q + "a": (H, D),
                      q + "A_log": (H,), q + "dt_bias": (H,), q + "norm": (m["vdim"],), q + "g": (vw, D),
                      q + "o": (D, vw)})
        else:
            R, r = m["kv_rank"], m["rot_dim"]
            s.update({q + "dq": (m["q_rank"], D), q + "dq.norm": (m["q_rank"],),
                      q + "uq": (H * (m["dim"] + r), m["q_rank"]), q + "uk": (H * m["dim"], R),
                      q + "uv": (H * m["vdim"], R), q + "sink": (H,), q + "o": (D, H * m["vdim"])})
            if m.get("kv_from") is None:
                s.update({q + "dkv": (R + r, D), q + "dkv.norm": (R,)})
        for n in (1, 2) if layer["mlp"] is not None else (1,):
            s.update({f"{p}norm{n}": (D,), f"{p}hc{n}.in": (S,), f"{p}hc{n}.out": (S,), f"{p}hc{n}.mix": (S, S)})
        if layer["mlp"] is not None:
            E, F = layer["mlp"]["router"]["experts"], layer["mlp"]["expert"]["ff"]
            s[p + "mlp.table"] = (V, layer["mlp"]["router"]["top"])
            for e in range(E):
                s.update({f"{p}mlp.e{e}.gate": (F, D), f"{p}mlp.e{e}.up": (F, D), f"{p}mlp.e{e}.down": (D, F)})
    return s


def random_weights(cfg, seed, sharp=1.0):
    """Random tensors (values that bfloat16 holds exactly; tables int32).  Matrices N(0, 1 / fan-in); ``sharp`` multiplies
    the latent layers' queries, so that the softmax sits on few keys."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    S = cfg["streams"]
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if leaf == "table":
            layer = int(name.split(".")[0][1:])
            E = cfg["layers"][layer]["mlp"]["router"]["experts"]
            w[name] = torch.rand((shape[0], E), generator=g).argsort(1)[:, :shape[1]].to(torch.int32)
            continue
        if name.endswith(("norm1", "norm2")) or name == "final.norm":
            t = 0.2 * torch.randn(shape, generator=g)
        elif leaf == "norm":
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif ".hc" in name:
            t = 0.4 * torch.randn(shape, generator=g)
            t = t / S + torch.eye(S) if leaf == "mix" else (t + 1.0) / (S if leaf == "in" else 1)
        elif leaf in ("A_log", "dt_bias", "sink", "b") and len(shape) == 1:
            t = 0.5 * torch.randn(shape, generator=g)
        elif leaf == "conv":
            t = torch.randn(shape, generator=g) / math.sqrt(shape[1])
        elif name == "embed":
            t = 0.5 * torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
            if leaf == "uq":
                t = t * sharp
        w[name] = t.to(torch.bfloat16).to(torch.float32)
    return w


def random_config(seed):
    """A configuration drawn at random: (config, page size).  Every size, count, constant and option that a configuration
    may state is drawn, the order of the layers too."""
    import random
    r = random.Random(seed)
    width = r.choice([32, 40, 52, 64, 96, 130])
    layers, own = [], []
    for i in range(r.randint(2, 6)):
        kind = r.choice(["attention", "delta", "latent", "latent"])
        window = r.choice([None, 1, 3, 7, 16, 33, 72])
        if kind == "attention":
            kv, dim = r.choice([1, 2, 4]), r.choice([8, 10, 16, 24, 40, 64, 72, 96, 128])
            mix = attend(kv * r.choice([1, 2, 3]), kv, dim, r.choice([6, 16, 32, 56, 64, 80, 128]),
                         dim ** -0.5 * r.choice([0.7, 1.0, 2.0]), window)
        elif kind == "delta":
            kv = r.choice([1, 2, 3])
            mix = delta(kv * r.choice([1, 2, 4]), kv, r.choice([4, 7, 16, 32, 64, 96]), r.choice([4, 9, 16, 32, 64, 130]),
                        r.randint(1, 6))
        else:
            heads, dim, vdim = r.randint(1, 6), r.choice([4, 9, 16, 32, 64]), r.choice([4, 8, 15, 64])
            q_rank, scale = r.choice([5, 8, 24, 64, 100]), r.choice([0.1, 0.2, 0.35])
            if own and r.random() < 0.6:
                j = r.choice(own)
                src = layers[j][0][1]
                sc = src["rot"].get("scaling")
                mix = latent(heads, dim, src["rot_dim"], vdim, src["kv_rank"], q_rank, scale, window, src["rot"]["base"],
                             tuple(sc.values()) if sc else None, kv_from=j)
            else:
                sc = None
                if r.random() < 0.6:
                    sc = (r.choice([1.5, 2.0, 8.0]), r.choice([8, 64, 512]), r.choice([4.0, 32.0]), r.choice([0.5, 1.0]))
                mix = latent(heads, dim, r.choice([2, 4, 8, 16, 32]), vdim, r.choice([8, 16, 20, 32, 64]), q_rank, scale,
                             window, r.choice([100.0, 10000.0, 1000000.0]), sc)
                own.append(i)
        ff = None
        if r.random() < 0.8:
            experts = r.choice([1, 2, 5, 8, 16])
            ff = moe(experts, r.randint(1, min(experts, 5)), r.choice([8, 13, 24, 64]))
        layers.append((mix, ff))
    cfg = model(r.randint(50, 200), width, r.choice([1, 2, 3, 4, 6]), r.choice([1e-5, 1e-6]), layers,
                scale=r.choice([1.0, 0.5, float(width) ** 0.5]))
    return cfg, r.choice([4, 8, 16])
