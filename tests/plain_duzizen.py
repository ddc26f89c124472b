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


# ---- configurations of the tests and random weights -----------------------------------------------------------
def memory(heads, dim, vdim, gate_cap):
    return ("mlstm", {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap})


def attention(heads, kv_heads, dim, scale, conv=0, window=None, keep_first=0, rot=None, scaling=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if conv:
        m["conv"] = conv
    if window is not None:
        m["mask"] = {"size": window, "keep_first": keep_first}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if scaling is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return m


def keep(heads, dim, vdim, decay, rot=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return m


def pair(left, right):
    return ("parallel", {"left": left, "right": right})


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(n, top, ff, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": n, "top": top}}


def model(vocab, width, eps, layers, bigram=None, side=None):
    """``layers``: [((type, mixer), mlp or None)]; ``bigram``: (buckets, mul_prev, mul_cur)."""
    j = {"architecture": "Duzizen", "vocab": vocab, "width": width, "norm": {"eps": eps},
         "layers": [{"type": t, "mixer": m, "mlp": q} for (t, m), q in layers]}
    if bigram is not None:
        j["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}
    if side is not None:
        j["token_side"] = {"dim": side}
    return j


# name -> (configuration, page size)
CONFIGS = {
    # a window of 21 over pages of 8 with three kept tokens, part of each head rotated with stretched wavelengths;
    # experts of which three are used; a layer without feed-forward
    "A": (model(90, 64, 1e-5, [
        (memory(3, 16, 24, 9.0), moe(6, 3, 24, 0.8)),
        (pair(attention(4, 2, 16, 0.3, conv=3, window=21, keep_first=3, rot=(8, 5000.0), scaling=(4.0, 1.0, 3.0, 64)),
              keep(2, 16, 8, (0.9, 0.997), rot=(16, 10000.0))), dense(72)),
        (memory(2, 8, 16, 4.0), None),
        (pair(attention(2, 1, 32, 0.2, conv=4, window=33, keep_first=9, rot=(32, 300.0)),
              keep(3, 12, 20, (0.5, 0.98, 1.0), rot=(4, 100.0))), moe(5, 1, 16, 1.5))],
        bigram=(61, 3, 11), side=10), 8),
    # sizes that are multiples of nothing; one head; no convolution, no pair table, no side input, no mask (every
    # earlier key), no rotation on the right
    "B": (model(71, 44, 1e-6, [
        (pair(attention(1, 1, 10, 0.4, rot=(6, 500.0)), keep(1, 6, 10, (0.95,))), dense(37)),
        (memory(1, 7, 5, 15.0), dense(64)),
        (pair(attention(3, 3, 20, 0.25, conv=1, window=1, keep_first=0), keep(2, 10, 6, (0.0, 0.9), rot=(2, 10.0))), None),
        (memory(5, 4, 12, 2.0), moe(3, 2, 11, 0.5))]), 4),
    # tensor-core head sizes, a kept token more than a page, a window shorter than a page, one that ends on a page
    "C": (model(130, 96, 1e-5, [
        (pair(attention(6, 2, 64, 0.125, conv=4, window=36, keep_first=17, rot=(32, 10000.0), scaling=(2.0, 1.0, 4.0, 32)),
              keep(2, 64, 64, (0.96, 0.999), rot=(64, 10000.0))), moe(8, 2, 32, 2.0)),
        (memory(2, 64, 64, 12.0), dense(128)),
        (pair(attention(2, 2, 128, 0.09, conv=2, window=5, keep_first=1, rot=(128, 1000.0)),
              keep(1, 128, 32, (0.99,), rot=(64, 500.0))), dense(64)),
        (memory(1, 128, 96, 8.0), moe(4, 4, 40, 1.0))], bigram=(31, 1, 7), side=16), 16),
}


def config(name):
    return CONFIGS[name]


def tensor_shapes(cfg):
    D, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, D), "head": (V, D), "final.norm": (D,), "final.norm.b": (D,)}
    b = (cfg.get("embedding") or {}).get("bigram")
    if b is not None:
        s["bigram"] = (b["buckets"] + 1, D)
    side = cfg.get("token_side")
    if side is not None:
        s["side.embed"] = (V, side["dim"] * len(cfg["layers"]))
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if layer["mlp"] is not None else ()):
            s[p + n] = s[p + n + ".b"] = (D,)
        q = p + "mix."
        if layer["type"] == "mlstm":
            H, qk, vw = m["heads"], m["heads"] * m["dim"], m["heads"] * m["vdim"]
            s.update({q + "q": (qk, D), q + "k": (qk, D), q + "v": (vw, D), q + "g": (vw, D), q + "o": (D, vw),
                      q + "norm": (vw,), q + "i": (H, D), q + "i.b": (H,), q + "f": (H, D), q + "f.b": (H,)})
        else:
            a, r = m["left"], m["right"]
            qw, kw = a["heads"] * a["dim"], a["kv_heads"] * a["dim"]
            s.update({q + "left.q": (qw, D), q + "left.k": (kw, D), q + "left.q.norm": (qw,), q + "left.k.norm": (kw,),
                      q + "left.o": (D, qw), q + "left.out": (D,), q + "right.out": (D,)})
            if a.get("conv"):
                s.update({q + "left.q.conv": (qw, a["conv"]), q + "left.k.conv": (kw, a["conv"])})
            qk, vw = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            s.update({q + "right.q": (qk, D), q + "right.k": (qk, D), q + "right.v": (vw, D), q + "right.g": (vw, D),
                      q + "right.o": (D, vw)})
        f = layer["mlp"]
        if f is not None and f["kind"] == "dense":
            s.update({p + "mlp.gate": (f["ff"], D), p + "mlp.up": (f["ff"], D), p + "mlp.down": (D, f["ff"])})
        elif f is not None:
            s[p + "mlp.router"] = (f["router"]["experts"], D)
            for e in range(f["router"]["experts"]):
                F = f["expert"]["ff"]
                s.update({p + f"mlp.e{e}.gate": (F, D), p + f"mlp.e{e}.up": (F, D), p + f"mlp.e{e}.down": (D, F)})
        if side is not None:
            s.update({p + "side.gate": (side["dim"], D), p + "side.proj": (D, side["dim"]), p + "side.norm": (D,)})
    return s


def random_weights(cfg, seed, sharp=1.0):
    """Random tensors (values that bfloat16 holds exactly).  Matrices N(0, 1 / fan-in); norm weights around one;
    ``sharp`` multiplies the attention layers' query norms, so that the softmax sits on few keys; the routers' rows are
    scaled up so that few choices are close."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if leaf == "b":
            t = 0.3 * torch.randn(shape, generator=g)
            if name.endswith(".f.b"):
                t = t + 3.0                      # remember for a while
        elif name.endswith((".conv",)):
            t = torch.randn(shape, generator=g) / math.sqrt(shape[1])
        elif len(shape) == 1:
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
            if name.endswith("left.q.norm"):
                t = t * sharp
        elif name in ("embed", "bigram", "side.embed"):
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
            if leaf == "router":
                t = t * 3.0
        w[name] = t.to(torch.bfloat16).to(torch.float32)
    return w


def random_config(seed):
    """A configuration drawn at random: (config, page size).  Every size, count, constant and option that a
    configuration may state is drawn, the order of the layers too."""
    import random
    r = random.Random(seed)
    width = r.choice([32, 40, 48, 64, 96])

    def rot_of(dim, scaled):
        dims = r.choice([d for d in (2, 4, 8, 16, 32, 64, dim // 2 * 2) if d <= dim])
        scaling = (r.choice([1.5, 4.0, 8.0]), 1.0, r.choice([2.0, 4.0]), r.choice([16, 64, 512])) if scaled else None
        return (dims, r.choice([100.0, 10000.0, 500000.0])), scaling

    layers = []
    for _ in range(r.randint(2, 5)):
        if r.random() < 0.45:
            mix = memory(r.choice([1, 2, 3, 4]), r.choice([4, 8, 16, 48, 64, 128]), r.choice([4, 8, 24, 32, 64, 96]),
                         r.choice([1.0, 5.0, 12.0]))
        else:
            kv, dim = r.choice([1, 2, 4]), r.choice([6, 8, 16, 24, 32, 48, 64, 128])
            rot, scaling = rot_of(dim, r.random() < 0.6) if r.random() < 0.85 else (None, None)
            left = attention(kv * r.choice([1, 2, 3]), kv, dim, dim ** -0.5 * r.choice([0.7, 1.0, 1.6]), conv=r.randint(0, 5),
                             window=r.choice([None, 1, 3, 7, 16, 33, 72]), keep_first=r.choice([0, 1, 4, 5, 16, 21]),
                             rot=rot, scaling=scaling)
            if "mask" not in left:
                left.pop("keep_first", None)
            H, d2 = r.choice([1, 2, 3]), r.choice([4, 8, 16, 48, 64, 128])
            right = keep(H, d2, r.choice([4, 8, 24, 32, 64, 96]), [r.choice([0.2, 0.9, 0.98, 0.999, 1.0]) for _ in range(H)],
                         rot=rot_of(d2, False)[0] if r.random() < 0.8 else None)
            mix = pair(left, right)
        n = r.choice([2, 4, 7, 16])
        mlp = r.choice([None, dense(r.choice([16, 30, 64, 100])), moe(n, r.randint(1, min(n, 3)), r.choice([8, 20, 32, 64]),
                                                                     r.choice([0.4, 1.0, 7.0]))])
        layers.append((mix, mlp))
    return model(r.randint(50, 200), width, r.choice([1e-5, 1e-6]), layers,
                 bigram=(r.choice([7, 31, 97]), r.randint(1, 40), r.randint(1, 40)) if r.random() < 0.7 else None,
                 side=r.choice([None, 3, 8, 24])), r.choice([4, 8, 16])
