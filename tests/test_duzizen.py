"""Duzizen in the engine against the plain implementation of ``plain_duzizen``.

Configuration, plan, kept pages and frequencies on the CPU; on the GPU the kernels of the design alone, each mixer and
each feed-forward as the only one of a model, then whole models under every way of cutting the work: whole prompts,
token-by-token decoding from the first token, portions down to two tokens, mixed batches with pages and state slots
that are used again; keys just inside and just outside a window, kept first tokens and the next ones, in prompts and
in decoding; a far token that decides through each recurrent state; the one in the denominator; the pair table
across portions; long decoding; greedy generation through the Python entry point and its scheduler; the programs.
"""
import copy
import json
import math
import os

import numpy as np
import pytest
import torch

import helpers
import plain_duzizen as plain

gpu = pytest.mark.gpu

TOL32 = 5e-5          # relative to the largest logit of the request
TOL16 = 8e-2
SHARP = {"float32": 3.0, "bfloat16": 1.5}   # the attention layers' query norms times this: the softmax sits on few keys


def write_model(path, name=None, cfg=None, seed=0, sharp=1.0, edit=None):
    from safetensors.torch import save_file
    if cfg is None:
        cfg, _ = plain.config(name)
    w = plain.random_weights(cfg, seed, sharp)
    if edit is not None:
        edit(w)
        w = {k: v.to(torch.bfloat16).to(torch.float32) for k, v in w.items()}
    os.makedirs(path, exist_ok=True)
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    return cfg, w


def engine_of(path, dtype, page, pool, max_requests=4, use_graphs=False, step_tokens=None):
    from ccinfer_b200.engine.engine import Engine, EngineOptions
    return Engine.from_model_dir(path, EngineOptions(
        dtype=dtype, page_size=page, kv_tokens=pool, max_requests=max_requests,
        max_tokens_per_step=step_tokens or pool, max_context=pool, use_graphs=use_graphs))


def compare(rows, ref, dtype, what):
    """32-bit: every row within TOL32.  bfloat16: norms on the sublayers' OUTPUTS divide by those outputs' size, so a
    token whose output nearly cancels has the rounding of that output magnified, and a close choice of experts may fall
    the other way: up to one row in 25 may lie beyond TOL16 while nine in ten lie within half of it."""
    if dtype == "float32":
        return helpers.compare(rows, ref, TOL32, what)
    errs = []
    for (rid, pos), row in rows.items():
        assert np.isfinite(row).all(), what
        errs.append(float(np.abs(row - ref[rid][pos]).max()) / max(1e-6, float(np.abs(ref[rid]).max())))
    errs = np.sort(np.array(errs))
    beyond = int((errs > TOL16).sum())
    assert beyond <= max(1, len(errs) // 25), f"{what}: {beyond} of {len(errs)} rows beyond {TOL16}"
    p90 = errs[int(0.9 * (len(errs) - 1))]
    assert p90 <= TOL16 / 2, f"{what}: nine rows in ten should lie within {TOL16 / 2:.1e}, not {p90:.2e}"
    return float(p90)


def requests_of(cfg, lengths, seed):
    rng = np.random.RandomState(seed)
    return {f"r{i}": rng.randint(0, cfg["vocab"], size=n).tolist() for i, n in enumerate(lengths)}


# ---------------------------------------------------------------------------------------------
# CPU: configuration, plan, frequencies, kept pages
# ---------------------------------------------------------------------------------------------
def test_config_is_read_written_and_refused():
    from ccinfer_b200.config.duzizen import DuzizenConfig
    from ccinfer_b200.config.registry import architecture_of
    from ccinfer_b200.errors import ModelConfigInvalid
    cfg, _ = plain.config("A")
    assert architecture_of(cfg).name == "Duzizen"
    c = DuzizenConfig.from_json(cfg)
    assert [l.type for l in c.layers] == ["mlstm", "parallel", "mlstm", "parallel"]
    assert c.pair.buckets == 61 and c.side_dim == 10 and c.layers[2].mlp is None
    left = c.layers[1].mixer.left
    assert (left.window, left.keep_first, left.conv, left.rot.dims, left.rot.scaling.high) == (21, 3, 3, 8, 3.0)
    assert c.layers[1].mixer.right.decay == (0.9, 0.997) and c.layers[0].mixer.gate_cap == 9.0
    assert c.layers[0].mlp.top == 3 and c.layers[0].mlp.limit == 0.8
    for name in plain.CONFIGS:
        full = DuzizenConfig.from_json(plain.config(name)[0])
        assert DuzizenConfig.from_json(full.to_json()) == full
    b = DuzizenConfig.from_json(plain.config("B")[0])
    assert b.pair is None and b.side_dim is None and b.layers[0].mixer.left.window is None
    assert b.layers[0].mixer.left.conv == 0 and b.layers[0].mixer.right.rot is None
    zero = copy.deepcopy(cfg)                      # whole numbers that may be zero
    zero["layers"][1]["mixer"]["left"]["conv"] = 0
    zero["layers"][1]["mixer"]["left"]["mask"]["keep_first"] = 0
    zero["embedding"]["bigram"]["mul_prev"] = 0
    assert DuzizenConfig.from_json(zero).layers[1].mixer.left.keep_first == 0
    for damage in (lambda j: j.pop("width"), lambda j: j["norm"].pop("eps"), lambda j: j["norm"].update(eps=0.0),
                   lambda j: j["embedding"]["bigram"].pop("mul_cur"), lambda j: j["layers"][0]["mixer"].pop("gate_cap"),
                   lambda j: j["layers"][0]["mixer"].update(gate_cap=0.0),
                   lambda j: j["layers"][1]["mixer"]["left"].pop("scale"),
                   lambda j: j["layers"][1]["mixer"]["left"].update(vdim=8),
                   lambda j: j["layers"][1]["mixer"]["left"].update(kv_heads=3),
                   lambda j: j["layers"][1]["mixer"]["left"].update(conv=-1),
                   lambda j: j["layers"][1]["mixer"]["left"]["mask"].pop("size"),
                   lambda j: j["layers"][1]["mixer"]["left"]["mask"].update(keep_first=-1),
                   lambda j: j["layers"][1]["mixer"]["left"]["rot"].update(dims=18),
                   lambda j: j["layers"][1]["mixer"]["left"]["rot"]["scaling"].pop("low"),
                   lambda j: j["layers"][1]["mixer"]["right"].update(decay=[0.9]),
                   lambda j: j["layers"][1]["mixer"]["right"].update(decay=[0.9, 1.5]),
                   lambda j: j["layers"][1]["mixer"].pop("right"), lambda j: j["layers"][1].update(type="attention"),
                   lambda j: j["layers"][0]["mlp"].pop("router"), lambda j: j["layers"][0]["mlp"]["router"].update(top=7),
                   lambda j: j["layers"][0]["mlp"]["expert"].pop("limit"), lambda j: j["layers"][1]["mlp"].pop("ff"),
                   lambda j: j["layers"][1]["mlp"].update(kind="gated"), lambda j: j["token_side"].pop("dim"),
                   lambda j: j.update(layers=[])):
        j = copy.deepcopy(cfg)
        damage(j)
        with pytest.raises(ModelConfigInvalid):
            DuzizenConfig.from_json(j)


def test_plan_names_every_tensor():
    from ccinfer_b200.architectures.duzizen import build_plan
    from ccinfer_b200.config.duzizen import DuzizenConfig
    for cfg in [plain.config(n)[0] for n in plain.CONFIGS] + [plain.random_config(s)[0] for s in range(40)]:
        plan = build_plan(DuzizenConfig.from_json(cfg))
        plan.validate()
        assert {s.name: tuple(s.shape) for s in plan.tensor_specs()} == plain.tensor_shapes(cfg)


def test_stretched_wavelengths():
    """Short wavelengths keep their frequency, long ones have it divided by the factor, between the two it grows with
    the wavelength's place; the package's table agrees with the plain one."""
    from ccinfer_b200.parts.position import RotaryHalf
    rot = {"dims": 16, "base": 700.0, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 256}}
    f = plain.rotary_frequencies(rot)
    plain_f = plain.rotary_frequencies({"dims": 16, "base": 700.0})
    assert f[0] == plain_f[0] and abs(f[-1] - plain_f[-1] / 8.0) < 1e-15
    mid = [i for i in range(8) if 64 < 2 * math.pi / plain_f[i] < 256]
    assert mid and all(plain_f[i] / 8.0 < f[i] < plain_f[i] for i in mid)
    r = RotaryHalf(16, 700.0, interleaved=True, wavelength_scaling=rot["scaling"])
    assert np.allclose(r.wavelength_frequencies(), f, rtol=1e-13)
    with pytest.raises(ValueError):
        RotaryHalf(16, 700.0, linear_scaling=1.0, wavelength_scaling=rot["scaling"])


def test_plain_softmax_with_one_in_the_denominator():
    s = torch.tensor([[-50.0, -60.0], [3.0, 1.0]], dtype=torch.float64)
    a = plain.softmax_plus_one(s, torch.ones(2, 2, dtype=torch.bool))
    e = torch.exp(s)
    assert torch.allclose(a, e / (1 + e.sum(-1, keepdim=True))) and a[0].sum() < 1e-20 < 0.9 < a[1].sum()


def test_kept_pages_stay_while_the_window_moves_on():
    """A group of a window of six with five kept tokens over pages of four: the two pages of the kept tokens stay,
    the others go when every later query has passed them; all come back when the request ends."""
    from ccinfer_b200.cache.manager import CacheManager, GroupSpec
    from ccinfer_b200.parts.base import CacheNeed
    m = CacheManager([GroupSpec(("kept", 5, 6, None), 6, 4, 12, None, 5), GroupSpec(("window", 6), 6, 4, 12)], 2, 32, 64)
    m.open("a")
    for n in (7, 2, 9, 1, 1, 8):
        m.reserve("a", n)
        m.commit("a")
        ctx = m.get("a").ctx_len
        for g, kept in ((0, 2), (1, 0)):
            table = m.get("a").tables[g]
            first = m.first_needed_page(g, ctx)
            assert [p >= 0 for p in table] == [i < kept or i >= first for i in range(len(table))], (ctx, g)
        m.check_consistency()
    assert m.get("a").pages_held(0) == m.get("a").pages_held(1) + 2
    m.close("a")
    assert all(p.used_pages == 0 for p in m.pools)
    need = CacheNeed.keys_and_values(2, 16, window=6, keep_first=5)
    assert need.group_key != CacheNeed.keys_and_values(2, 16, window=6).group_key
    assert CacheNeed.keys_and_values(2, 16, keep_first=5).group_key == ("all",)   # without a mask everything stays


def test_parts_refuse_what_they_do_not_compute():
    from ccinfer_b200 import kernels
    from ccinfer_b200.errors import Unsupported
    from ccinfer_b200.parts import ExponentialGateMemory, GroupedQueryAttention, MixtureOfExperts, NoPosition, Retention
    names = {k: k for k in ("q", "k", "v", "o", "g", "norm", "i", "i_bias", "f", "f_bias")}
    with pytest.raises(Unsupported):
        Retention(16, 2, 8, 8, [0.5], 1e-5, names)
    with pytest.raises(Unsupported):
        ExponentialGateMemory(16, 2, 300, 8, 1.0, 1e-5, names)
    with pytest.raises(Unsupported):
        GroupedQueryAttention(16, 2, 1, 16, NoPosition(), names, value_dim=32, keys_as_values=True)
    with pytest.raises(Unsupported):
        GroupedQueryAttention(16, 2, 1, 16, NoPosition(), dict(names, sink="s"), sink_score=0.0)
    with pytest.raises(Unsupported):
        MixtureOfExperts(16, 4, 2, 8, {}, activation="relu2", weight_on_input=True)
    with pytest.raises(Unsupported):
        kernels.GluAct.clamped(0.0, 1.0, 1.0)


# ---------------------------------------------------------------------------------------------
# GPU: the kernels alone
# ---------------------------------------------------------------------------------------------
@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D", [48, 77, 1000, 2048, 4096, 6000, 9000])
@pytest.mark.parametrize("post,nxt", [("layer", "layer"), ("rms", "layer"), (None, "rms"), ("layer", None)])
def test_norm_chain(dtype, D, post, nxt):
    """Two sublayers' norms, the sum and the next norm, with a pair and rows to add; the deviations' variance under a
    large common offset; single rows picked by index, the stream untouched."""
    from ccinfer_b200 import kernels
    g = torch.Generator().manual_seed(D)
    T, eps = (200 if D >= 1000 and post == "layer" else 5), 1e-5    # (many rows run with other launch shapes)
    rnd = lambda *s: torch.randn(*s, generator=g)
    h, add = 3 * rnd(T, D) + 40.0, rnd(T, D)
    a, b = (2 * rnd(T, D) + 1.0).to(dtype), rnd(T, D).to(dtype)
    w = [1 + 0.3 * rnd(D) for _ in range(6)]

    def norm(kind, x, wt, bs):
        if kind is None:
            return x
        return plain.layer_norm(x, wt.double(), bs.double(), eps) if kind == "layer" else plain.rms_unit(x, eps) * wt.double()

    def spec(kind, wt, bs):
        return None if kind is None else kernels.NormSpec(kind, wt.cuda(), bs.cuda() if kind == "layer" else None, eps)

    tol = 2e-5 if dtype == torch.float32 else 4e-2
    for pair in (False, True):
        d = a.double()
        if pair:
            d = 0.5 * plain.rms_unit(a.double(), eps) * w[4].double() + 0.7 * plain.rms_unit(b.double(), eps) * w[5].double()
        want_h = h.double() + 0.8 * norm(post, d, w[0], w[1]) + add.double()
        want_y = norm(nxt, want_h, w[2], w[3])
        hd, y = h.cuda(), torch.empty(T, D, dtype=dtype, device="cuda")
        args = (b.cuda(), w[4].cuda(), w[5].cuda(), 0.5, 0.7, eps) if pair else None
        kernels.norm_chain(hd, a.cuda(), spec(post, w[0], w[1]), spec(nxt, w[2], w[3]), y=y, mult=0.8, add=add.cuda(),
                           pair=args)
        assert (hd.cpu().double() - want_h).abs().max() < 3e-5
        scale = max(1.0, float(want_y.abs().max())) if nxt is None else 4.0
        assert (y.cpu().double() - want_y).abs().max() < tol * scale, (pair, float((y.cpu().double() - want_y).abs().max()))
    if nxt is not None:
        idx = torch.tensor([3, 0, 3], dtype=torch.int32).cuda()
        hd, y = h.cuda(), torch.zeros(3, D, dtype=dtype, device="cuda")
        kernels.norm_chain(hd, a.cuda(), None, spec(nxt, w[2], w[3]), y=y, row_idx=idx)
        want = norm(nxt, h.double() + a.double(), w[2], w[3])[[3, 0, 3]]
        assert (y.cpu().double() - want).abs().max() < 4 * tol and torch.equal(hd.cpu(), h)


@gpu
def test_norm_chain_reports_a_bad_row():
    from ccinfer_b200 import kernels
    h, y = torch.randn(3, 64, device="cuda"), torch.ones(2, 64, device="cuda")
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    one = torch.ones(64, device="cuda")
    kernels.norm_chain(h, nxt=kernels.NormSpec("layer", one, one, 1e-5), y=y, status=status,
                       row_idx=torch.tensor([1, 3], dtype=torch.int32, device="cuda"))
    assert int(status.item()) == kernels.ST_BAD_ROW and (y[1] == 0).all() and (y[0] != 0).any()


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("F,block", [(64, 64), (128, 64), (37, 0)])
def test_gelu_gate_kernel(dtype, F, block):
    from ccinfer_b200 import kernels
    g = torch.Generator().manual_seed(F)
    gate, up = (4 * torch.randn(9, F, generator=g)).to(dtype), torch.randn(9, F, generator=g).to(dtype)
    gate[0, :4] = torch.tensor([-60.0, 60.0, 0.0, -8.0])
    gu = torch.cat([gate, up], 1)
    if block:
        gu = torch.cat([x for i in range(0, F, block) for x in (gate[:, i:i + block], up[:, i:i + block])], 1)
    act = torch.empty(9, F, dtype=dtype, device="cuda")
    kernels.gated_act(act, gu.contiguous().cuda(), block, kernels.GluAct.gelu_tanh())
    want = plain.gelu_tanh(gate.double()) * up.double()
    assert (act.cpu().double() - want).abs().max() < (1e-5 if dtype == torch.float32 else 1e-2) * want.abs().max()


@gpu
@pytest.mark.parametrize("kind,M", [("tc", 3), ("fewrows", 7), ("pair", 300)])
def test_gelu_gate_as_a_products_epilogue(kind, M):
    from ccinfer_b200 import kernels
    g = torch.Generator().manual_seed(M)
    F, K = 256, 2048
    x = torch.randn(M, K, generator=g).bfloat16()
    wg, wu = ((torch.randn(F, K, generator=g) / math.sqrt(K)).bfloat16() for _ in range(2))
    act = torch.empty(M, F, dtype=torch.bfloat16, device="cuda")
    kernels.gemm_glu_bf16(act, x.cuda(), kernels.interleave_gate_up(wg.cuda(), wu.cuda(), 64), kernels.GluAct.gelu_tanh(), kind)
    want = plain.gelu_tanh(x.double() @ wg.double().T) * (x.double() @ wu.double().T)
    assert (act.cpu().double() - want).abs().max() < 2e-2 * want.abs().max()


def _paged(x, page, n_pages, perm):
    """x [T, heads, hd] of ONE request into a cache [n_pages, heads, page, hd] with its pages at ``perm``."""
    T, Hh, hd = x.shape
    cache = torch.zeros(n_pages, Hh, page, hd, dtype=x.dtype)
    for t in range(T):
        cache[perm[t // page], :, t % page] = x[t]
    return cache


@gpu
@pytest.mark.parametrize("which", ["split float", "split", "decode_mma", "decode_tma", "prefill_mma", "prefill_tc",
                                   "prefill_tc one head"])
@pytest.mark.parametrize("window,keep_first", [(40, 3), (40, 17), (7, 1), (1, 70), (64, 64), (200, 9), (33, 300)])
def test_kept_first_keys_in_every_attention_kernel(which, window, keep_first):
    """A sequence of 330 tokens over shuffled pages of which the pages that no query needs any more do not exist:
    the window's keys, the kept ones and the sink of score zero, each query row."""
    from ccinfer_b200 import kernels
    dtype = torch.float32 if which == "split float" else torch.bfloat16
    nq, nkv, hd, T, page = 4, 2, 64, 330, 16
    g = torch.Generator().manual_seed(window + keep_first)
    q = torch.randn(T, nq, hd, generator=g).to(dtype)
    k, v = (torch.randn(T, nkv, hd, generator=g).to(dtype) for _ in range(2))
    sink = torch.zeros(nq)
    scale, first = 0.2, 0
    decode = which.startswith(("split", "decode"))
    # rows first .. T - 1 are asked for: decode kernels as single rows of the late part, the others as one portion
    first = 250 if decode else 180
    n_pages = 30
    perm = torch.randperm(n_pages, generator=g).tolist()[:-(-T // page)]
    s = torch.einsum("ihd,jhd->hij", q.double(), k.double().repeat_interleave(2, 1)) * scale
    a = plain.softmax_plus_one(s, plain.visible(T, {"size": window, "keep_first": keep_first})[None])
    want = torch.einsum("hij,jhd->ihd", a, v.double().repeat_interleave(2, 1))[first:]
    bt = torch.full((1, 32), -1, dtype=torch.int32)
    gone = set()
    for lp, pg in enumerate(perm):
        lo, hi = lp * page, lp * page + page - 1
        if hi < first - window + 1 and lo >= keep_first:
            gone.add(pg)                        # given back: no entry, and rubbish in its place
        else:
            bt[0, lp] = pg
    kc, vc = _paged(k, page, n_pages, perm), _paged(v, page, n_pages, perm)
    for pg in gone:
        kc[pg] = 1e4
        vc[pg] = 1e4
    kc, vc, bt = kc.cuda(), vc.cuda(), bt.cuda()
    n = T - first
    qd = q[first:].contiguous().cuda()
    out = torch.full((n, nq, hd), float("nan"), dtype=dtype, device="cuda")
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    extra = {"sink": sink.cuda(), "keep": keep_first, "status": status}
    if decode:
        pos = torch.arange(first, T, dtype=torch.int32).cuda()
        eot = torch.zeros(n, dtype=torch.int32).cuda()
        fn = {"split": kernels.attention_split, "split float": kernels.attention_split,
              "decode_mma": kernels.attention_decode_mma, "decode_tma": kernels.attention_decode_tma}[which]
        for splits in (1, 3):
            acc = torch.empty(n * nq * splits * hd, device="cuda") if splits > 1 else None
            ml = torch.empty(n * nq * splits * 2, device="cuda") if splits > 1 else None
            out.fill_(float("nan"))
            fn(qd, kc, vc, out, acc, ml, pos, eot, bt, 1, 0, n, window, scale, splits, **extra)
            err = (out.cpu().double() - want).abs().max()
            assert err < (2e-5 if dtype == torch.float32 else 3e-2), (splits, float(err))
    else:
        cu = torch.tensor([0, n], dtype=torch.int32).cuda()
        pos0 = torch.tensor([first], dtype=torch.int32).cuda()
        if which == "prefill_mma":
            kernels.attention_prefill_mma(qd, kc, vc, out, cu, pos0, bt, 0, 1, n, window, scale, **extra)
        else:
            kernels.attention_prefill_tc_single_head(which.endswith("one head"))
            try:
                kernels.attention_prefill_tc(qd, kc, vc, out, cu, pos0, bt, 0, 1, n, window, scale, **extra)
            finally:
                kernels.attention_prefill_tc_single_head(False)
        err = (out.cpu().double() - want).abs().max()
        assert err < 3e-2, float(err)
    assert int(status.item()) == 0


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nq,nkv,hd,n_real,taps,norm,rot", [
    (4, 2, 16, 16, 3, True, True), (1, 1, 32, 20, 1, True, True), (6, 2, 64, 64, 4, True, False),
    (2, 2, 64, 60, 2, True, True), (2, 1, 16, 16, 1, True, True),
    (32, 8, 128, 128, 4, True, True), (3, 3, 48, 44, 6, False, True), (12, 12, 256, 256, 2, True, True)])
def test_qk_rows_kernel(dtype, nq, nkv, hd, n_real, taps, norm, rot):
    """Queries, keys and values from the product's rows: a request that goes on with several tokens, one that brings
    one (its state is moved on here), one that starts, a padding row; then the others' state."""
    from ccinfer_b200 import kernels
    g = torch.Generator().manual_seed(hd + taps)
    C, eps, page = (nq + nkv) * hd, 1e-5, 8
    rnd = lambda *s: torch.randn(*s, generator=g)
    real = (torch.arange(C) % hd < n_real).float()
    many = 700 if hd in (16, 64) else 3             # (many tokens: several a block)
    counts, starts = [1, 5, many], [6, 9, 0]        # single-token entries first, as a step lists them
    full = [(rnd(s + n, C) * real).to(dtype) for s, n in zip(starts, counts)]
    conv = (rnd(taps, C) if taps > 1 else None)
    qw, kw = (1 + 0.3 * rnd(nq * hd)), (1 + 0.3 * rnd(nkv * hd))
    inv = torch.rand(hd // 2, generator=g)
    inv[hd // 4:] = 0.0
    rows = torch.cat([f[s:] for f, s in zip(full, starts)] + [torch.zeros(1, C, dtype=dtype)])
    T = rows.shape[0]
    keep = taps - 1
    slots = [3, 0, 2]
    state = torch.zeros(4, max(keep, 1), C, dtype=dtype)
    if keep:
        for f, s, sl in zip(full, starts, slots):
            tail = torch.cat([torch.zeros(keep, C, dtype=dtype), f[:s]])[-keep:]
            state[sl] = tail
    wide = torch.zeros(T, C + 8, dtype=dtype)
    wide[:, :C] = rows
    sd = state.cuda()
    q_out = torch.zeros(T, nq, hd, dtype=dtype, device="cuda")
    kc, vc = (torch.zeros(-(-(3 * T + 4) // page), nkv, page, hd, dtype=dtype, device="cuda") for _ in range(2))
    slot_map = torch.arange(T, dtype=torch.int32) * 3 + 1
    slot_map[-1] = -1
    pos = torch.tensor([6] + list(range(9, 14)) + list(range(many)) + [0], dtype=torch.int32)
    eot = torch.tensor([0] + [1] * 5 + [2] * many + [-1], dtype=torch.int32)
    cu = torch.tensor([0, 1, 6, 6 + many], dtype=torch.int32)
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    wd = None if conv is None else conv.to(dtype).cuda()
    kernels.qk_rows(wide.cuda()[:, :C + 8], q_out, kc, vc, wd, taps, sd if keep else None, qw.cuda() if norm else None,
                    kw.cuda() if norm else None, eps, n_real, inv.cuda() if rot else None, pos.cuda(), slot_map.cuda(),
                    eot.cuda(), cu.cuda(), torch.tensor(slots, dtype=torch.int32).cuda(), 3, status=status)
    if keep:
        kernels.conv_state_rows(wide.cuda()[:, :C], taps, C, sd, cu.cuda(), torch.tensor(slots, dtype=torch.int32).cuda(), 1, 2)
    t = 0
    tol = 2e-5 if dtype == torch.float32 else 4e-2
    for f, s, n in zip(full, starts, counts):
        u = f.double()
        if conv is not None:
            u = plain.causal_conv(u, conv.to(dtype).double().T)
        for i in range(s, s + n):
            qv, kv = u[i, :nq * hd], u[i, nq * hd:]
            qn, kn = qv, kv
            if norm:
                qn = qv / torch.sqrt((qv * qv).sum() / (nq * n_real) + eps) * qw.double()
                kn = kv / torch.sqrt((kv * kv).sum() / (nkv * n_real) + eps) * kw.double()
            out = []
            for x in (qn.view(nq, hd), kn.view(nkv, hd)):
                a, b = x[:, :hd // 2], x[:, hd // 2:]
                ang = (i * inv.double()) if rot else torch.zeros(hd // 2, dtype=torch.float64)
                out.append(torch.cat([a * ang.cos() - b * ang.sin(), b * ang.cos() + a * ang.sin()], 1))
            sm = int(slot_map[t])
            got = (q_out[t], kc[sm // page, :, sm % page], vc[sm // page, :, sm % page])
            for x, want in zip(got, (out[0], out[1], kv.view(nkv, hd))):
                # (a float angle at position i is off by up to i * 6e-8)
                assert (x.cpu().double() - want).abs().max() < (tol + 2e-7 * i) * max(1.0, float(want.abs().max())), t
            t += 1
    if keep:
        for f, sl in zip(full, slots):
            want = torch.cat([torch.zeros(keep, C, dtype=dtype), f])[-keep:]
            assert torch.equal(sd[sl].cpu(), want)
    assert int(status.item()) == 0


def _gates(zi, zf, bi, bf, cap, m0):
    """Step by step, float64: decay, write factor and exp(-m) of every token, and the last m."""
    i = cap * torch.tanh((zi.double() + bi.double()) / cap)
    f = plain.log_sigmoid(cap * torch.tanh((zf.double() + bf.double()) / cap))
    m, out = m0.double(), []
    for t in range(i.shape[0]):
        new = torch.maximum(f[t] + m, i[t])
        out.append((torch.exp(f[t] + m - new), torch.exp(i[t] - new), torch.exp(-new)))
        m = new
    return [torch.stack(x) for x in zip(*out)], m


@gpu
def test_memory_gates_kernel():
    """Running maxima over portions of 1, 2, 31, 32, 33, 300 and 700 tokens from a state that earlier tokens left."""
    from ccinfer_b200 import kernels
    g = torch.Generator().manual_seed(0)
    H, cap, counts = 5, 6.0, [1, 2, 31, 32, 33, 300, 700]
    T = sum(counts)
    z = 8 * torch.randn(T, 2 * H + 3, generator=g)
    bi, bf = torch.randn(H, generator=g), torch.randn(H, generator=g) + 2
    m0 = torch.randn(9, H, generator=g)
    slots = [4, 0, 8, 2, 1, 7, 3]
    cu = torch.tensor([0] + list(np.cumsum(counts)), dtype=torch.int32)
    md = m0.cuda()
    outs = [torch.zeros(T, H, device="cuda") for _ in range(3)]
    kernels.memory_gates(z.cuda(), bi.cuda(), bf.cuda(), cap, md, cu.cuda(), torch.tensor(slots, dtype=torch.int32).cuda(),
                         *outs, len(counts), H)
    for e, n in enumerate(counts):
        r = slice(int(cu[e]), int(cu[e]) + n)
        want, m = _gates(z[r, :H], z[r, H:2 * H], bi, bf, cap, m0[slots[e]])
        for x, y in zip(outs, want):
            assert (x[r].cpu().double() - y).abs().max() < 2e-5 * max(1.0, float(y.abs().max())), n
        assert (md[slots[e]].cpu().double() - m).abs().max() < 1e-5
    untouched = [s for s in range(9) if s not in slots]
    assert torch.equal(md.cpu()[untouched], m0[untouched])


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dk,dv,rot,ones", [(3, 16, 24, 16, False), (2, 64, 64, 32, False), (1, 7, 5, 0, True), (5, 12, 128, 4, True)])
def test_memory_prepare_kernel(dtype, H, dk, dv, rot, ones):
    from ccinfer_b200 import kernels
    g = torch.Generator().manual_seed(dk)
    T = 9
    ok, ov = H * dk + 3, 2 * H * dk + 3
    proj = torch.randn(T, ov + H * dv + 2, generator=g).to(dtype)
    inv = torch.rand(max(rot // 2, 1), generator=g)
    pos = torch.randint(0, 500, (T,), generator=g, dtype=torch.int32)
    qn, kn = (torch.empty(T, H, dk, device="cuda") for _ in range(2))
    vv = torch.empty(T, H, dv + (1 if ones else 0), device="cuda")
    kernels.memory_prepare(proj.cuda(), (0, ok, ov), inv.cuda() if rot else None, rot, pos.cuda(), qn, kn, vv, H, dk, dv,
                           0.7, 0.3, ones=ones)
    ang = pos.double()[:, None] * inv.double()[None]
    for got, off, mult in ((qn, 0, 0.7), (kn, ok, 0.3)):
        x = proj[:, off:off + H * dk].double().view(T, H, dk).clone()
        if rot:
            a, b = x[..., :rot // 2].clone(), x[..., rot // 2:rot].clone()
            c, s = ang.cos()[:, None], ang.sin()[:, None]
            x[..., :rot // 2], x[..., rot // 2:rot] = a * c - b * s, b * c + a * s
        assert (got.cpu().double() - mult * x).abs().max() < 2e-4
    want = proj[:, ov:ov + H * dv].double().view(T, H, dv)
    if ones:
        want = torch.cat([want, torch.ones(T, H, 1, dtype=torch.float64)], -1)
    assert torch.equal(vv.cpu().double(), want)


def _recurrence(q, k, v, decay, put, S):
    """One request, float64: q, k [T, H, dk], v [T, H, dv], decay and put [T, H], S [H, dv, dk]; read-outs and last S."""
    out = []
    for t in range(q.shape[0]):
        S = decay[t][:, None, None] * S + put[t][:, None, None] * v[t][:, :, None] * k[t][:, None, :]
        out.append(torch.einsum("hvk,hk->hv", S, q[t]))
    return torch.stack(out), S


@gpu
@pytest.mark.parametrize("H,dk,dv,ones,split", [(2, 64, 32, True, False), (1, 128, 48, True, False), (3, 128, 64, False, True),
                                                (2, 64, 16, False, True), (26, 64, 128, True, False),
                                                (2, 128, 32, True, True)])
def test_memory_chunks_kernel(H, dk, dv, ones, split):
    """Chunks of 64 tokens on tensor cores, portions of 2, 63, 64, 65, 130 and 300 tokens from states that earlier
    tokens left, decays from nothing kept to everything, one far token that decides: to about 2^-15 of the result."""
    from ccinfer_b200 import kernels
    g = torch.Generator().manual_seed(H + dk + dv)
    counts, slots = [1, 2, 63, 64, 65, 130, 300], [0, 3, 6, 1, 7, 2, 5]
    T, dvo = sum(counts), dv + (1 if ones else 0)
    rnd = lambda *s: torch.randn(*s, generator=g)
    la = -torch.exp(2.5 * rnd(T, H) - 4.0)
    la[::37] = -40.0
    la[:, 0] = -1e-4
    lb = rnd(T, H)
    qf, kf = rnd(T, H * dk), rnd(T, H * dk)
    kf[-200] = 30 * rnd(H * dk)
    qf[-1] = kf[-200]                                  # the last query asks for a token 199 places back
    q_hi, k_hi = qf.bfloat16(), kf.bfloat16()
    q_lo, k_lo = ((x - h.float()).bfloat16() for x, h in ((qf, q_hi), (kf, k_hi)))
    wide = torch.zeros(T, H * dk + H * dv + 8, dtype=torch.bfloat16)
    wide[:, :H * dv] = rnd(T, H * dv).bfloat16()
    q, k = (x.double().view(T, H, dk) for x in ((qf, kf) if split else (q_hi, k_hi)))
    v = wide[:, :H * dv].double().view(T, H, dv)
    if ones:
        v = torch.cat([v, torch.ones(T, H, 1, dtype=torch.float64)], -1)
    S0 = rnd(8, H, dvo, dk)
    cu = torch.tensor([0] + list(np.cumsum(counts)), dtype=torch.int32)
    Sd = S0.cuda()
    out = torch.full((T, H, dvo), float("nan"), device="cuda")
    dev = lambda x: x.cuda()
    kernels.memory_chunks((dev(q_hi), dev(q_lo) if split else None), (dev(k_hi), dev(k_lo) if split else None), dev(wide),
                          dev(la), dev(lb) if ones else None, Sd, out, dev(cu), dev(torch.tensor(slots, dtype=torch.int32)),
                          1, len(counts) - 1, H, dk, dv, 0.7)
    put = torch.exp(lb.double()) if ones else torch.ones(T, H, dtype=torch.float64)
    for e in range(1, len(counts)):
        r = slice(int(cu[e]), int(cu[e + 1]))
        want, S = _recurrence(q[r], k[r], v[r], torch.exp(la.double())[r], put[r], S0[slots[e]].double())
        want = 0.7 * want
        err = (out[r].cpu().double() - want).abs().amax((0, 2)) / want.abs().amax((0, 2))
        assert err.max() < 1e-4, (counts[e], err)
        err = (Sd[slots[e]].cpu().double() - S).abs().amax((1, 2)) / S.abs().amax((1, 2))
        assert err.max() < 1e-4, (counts[e], err)
    assert torch.equal(Sd[0].cpu(), S0[0]) and torch.equal(Sd[4].cpu(), S0[4])    # entry 0 and a free slot: untouched


@gpu
def test_rotated_rows_as_two_bfloat16():
    from ccinfer_b200 import kernels
    g = torch.Generator().manual_seed(5)
    for H, dk, rot in ((2, 64, 64), (3, 128, 32), (1, 64, 0), (2, 20, 12)):
        T, ok = 7, H * dk + 6
        proj = torch.randn(T, ok + H * dk, generator=g).bfloat16()
        inv = torch.rand(max(rot // 2, 1), generator=g)
        pos = torch.randint(0, 300, (T,), generator=g, dtype=torch.int32)
        q, k = ([torch.empty(T, H * dk, dtype=torch.bfloat16, device="cuda") for _ in range(2)] for _ in range(2))
        kernels.memory_rotate_split(proj.cuda(), (0, ok), inv.cuda() if rot else None, rot, pos.cuda(), q, k, H, dk, 1.0, 0.3)
        qn, kn = (torch.empty(T, H, dk, device="cuda") for _ in range(2))
        vv = torch.empty(T, H, 1, device="cuda")
        kernels.memory_prepare(proj.cuda(), (0, ok, 0), inv.cuda() if rot else None, rot, pos.cuda(), qn, kn, vv, H, dk, 1,
                               1.0, 0.3)
        for (hi, lo), want in ((q, qn), (k, kn)):
            err = (hi.double() + lo.double() - want.view(T, -1).double()).abs().max() / want.abs().max()
            assert err < 2.0 ** -16, (H, dk, rot, float(err))


@gpu
@pytest.mark.parametrize("dtypes", [("float32", "float32"), ("float32", "bfloat16"), ("bfloat16", "bfloat16")])
@pytest.mark.parametrize("H,dk,dv,rot,ones", [(3, 16, 24, 16, False), (2, 64, 64, 32, False), (1, 7, 5, 0, True),
                                              (5, 128, 96, 0, True), (2, 256, 130, 128, False), (2, 36, 20, 4, True)])
def test_memory_step_kernel(dtypes, H, dk, dv, rot, ones):
    """One token of each of three requests (and a padding entry) in one kernel, against the gates, the rotation, the
    recurrence and the output one after another."""
    from ccinfer_b200 import kernels
    ti, to = (getattr(torch, d) for d in dtypes)
    g = torch.Generator().manual_seed(dk + dv)
    rnd = lambda *s: torch.randn(*s, generator=g)
    B, dvo, eps, cap = 4, dv + (1 if ones else 0), 1e-5, 7.0
    ok, ov = H * dk + 1, 2 * H * dk + 2
    og = ov + H * dv + 3
    proj = rnd(B, og + H * dv).to(ti)
    z = 3 * rnd(B, 2 * H + 1)
    bi, bf, m0 = rnd(H), rnd(H) + 2, rnd(6, H)
    decay = torch.rand(H, generator=g)
    S0 = rnd(6, H, dvo, dk)
    w = 1 + 0.2 * rnd(H * dv) if ones else None
    inv = torch.rand(max(rot // 2, 1), generator=g)
    pos = torch.tensor([0, 17, 230, 0], dtype=torch.int32)
    slots = torch.tensor([4, 0, 2, -1], dtype=torch.int32)
    Sd, md = S0.cuda(), m0.cuda()
    y = torch.zeros(B, H * dv, dtype=to, device="cuda")
    gates = (z.cuda(), 0, H, bi.cuda(), bf.cuda(), cap, md) if ones else decay.cuda()
    kernels.memory_step(y, proj.cuda(), (0, ok, ov, og), gates, Sd, inv.cuda() if rot else None, rot, pos.cuda(),
                        torch.arange(B + 1, dtype=torch.int32).cuda(), slots.cuda(), B, H, dk, dv, 0.6, 0.4, eps,
                        weight=None if w is None else w.cuda(), den_eps=1e-6 if ones else 0.0, silu_gate=not ones, ones=ones)
    p = proj.double()
    for b in range(3):
        q, k = p[b, :H * dk].view(H, dk).clone(), p[b, ok:ok + H * dk].view(H, dk).clone()
        if rot:
            ang = float(pos[b]) * inv.double()
            for x in (q, k):
                u, v = x[:, :rot // 2].clone(), x[:, rot // 2:rot].clone()
                x[:, :rot // 2], x[:, rot // 2:rot] = u * ang.cos() - v * ang.sin(), v * ang.cos() + u * ang.sin()
        v = p[b, ov:ov + H * dv].view(H, dv)
        sl = int(slots[b])
        if ones:
            v = torch.cat([v, torch.ones(H, 1, dtype=torch.float64)], -1)
            (a, put, fl), m = _gates(z[b:b + 1, :H], z[b:b + 1, H:2 * H], bi, bf, cap, m0[sl])
            assert (md[sl].cpu().double() - m).abs().max() < 1e-5
        else:
            a, put = decay.double()[None], torch.ones(1, H, dtype=torch.float64)
        o, S = _recurrence(0.6 * q[None], 0.4 * k[None], v[None], a, put, S0[sl].double())
        assert (Sd[sl].cpu().double() - S).abs().max() < 3e-4 * max(1.0, float(S.abs().max()))
        x = o[0][:, :dv]
        if ones:
            x = x / (torch.maximum(o[0][:, dv].abs(), fl[0]) + 1e-6)[:, None]
        x = plain.rms_unit(x, eps).reshape(-1) * (w.double() if ones else 1.0)
        gate = p[b, og:og + H * dv]
        want = x * (torch.sigmoid(gate) if ones else plain.silu(gate))
        assert (y[b].cpu().double() - want).abs().max() < (3e-4 if to == torch.float32 else 2e-2) * max(1.0, float(want.abs().max()))
    assert (y[3] == 0).all()
    for sl in (1, 3, 5):
        assert torch.equal(Sd[sl].cpu(), S0[sl]) and torch.equal(md[sl].cpu(), m0[sl])


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dv", [(3, 24), (2, 64), (1, 5), (4, 300)])
def test_memory_output_kernel(dtype, H, dv):
    from ccinfer_b200 import kernels
    g = torch.Generator().manual_seed(dv)
    T, eps = 7, 1e-5
    gate = torch.randn(T, H * dv + 5, generator=g).to(dtype)
    w = 1 + 0.2 * torch.randn(H * dv, generator=g)
    for floor in (None, torch.rand(T, H, generator=g) * 2):
        o = torch.randn(T, H, dv + (0 if floor is None else 1), generator=g)
        for silu, weight in ((True, None), (False, w)):
            y = torch.empty(T, H * dv, dtype=dtype, device="cuda")
            kernels.memory_output(y, o.cuda(), gate.cuda(), H, dv, eps, weight=None if weight is None else weight.cuda(),
                                  floor=None if floor is None else floor.cuda(), den_eps=1e-6, silu_gate=silu)
            x = o.double()[..., :dv]
            if floor is not None:
                x = x / (torch.maximum(o.double()[..., dv].abs(), floor.double()) + 1e-6)[..., None]
            x = plain.rms_unit(x, eps).reshape(T, H * dv)
            if weight is not None:
                x = x * weight.double()
            gd = gate.double()[:, :H * dv]
            want = x * (plain.silu(gd) if silu else torch.sigmoid(gd))
            assert (y.cpu().double() - want).abs().max() < (1e-5 if dtype == torch.float32 else 2e-2) * max(1.0, float(want.abs().max()))


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,top,F,sparse", [(6, 2, 32, False), (6, 2, 32, True), (16, 1, 64, True), (5, 5, 24, True),
                                            (16, 1, 64, False), (3, 2, 11, False)])
def test_experts_weighted_on_their_input(tmp_path, dtype, n, top, F, sparse, monkeypatch):
    """The mixture as a part of a model, every expert on every token or only the chosen ones (tiles of 16 rows and,
    in bfloat16 from some rows an expert on, tcgen05 tiles), with a limit that cuts many gates and ups."""
    from ccinfer_b200.parts import MixtureOfExperts
    if sparse:
        monkeypatch.setattr(MixtureOfExperts, "SPARSE_MIN_WEIGHTS", 1)
    cfg = plain.model(60, 64, 1e-5, [(plain.memory(1, 8, 8, 5.0), plain.moe(n, top, F, 0.6))])
    d = str(tmp_path / "moe")
    cfg, w = write_model(d, cfg=cfg, seed=n + top)
    reqs = requests_of(cfg, [1, 5, 40, 150], 1)
    ref = {rid: plain.forward(cfg, w, t).numpy() for rid, t in reqs.items()}
    for steps in (helpers.trace_whole(reqs), helpers.trace_mixed(reqs, max_live=3, seed=2)):
        eng = engine_of(d, dtype, 8, helpers.max_live_tokens(steps, round_to=64))
        assert eng.plan.layers[0].ffn.use_sparse == (sparse and (dtype == "float32" or F % 8 == 0))
        compare(helpers.replay(eng, steps), ref, dtype, f"experts {n} {top} {F} {dtype}")


# ---------------------------------------------------------------------------------------------
# GPU: each mixer as the only layer of a model
# ---------------------------------------------------------------------------------------------
ALONE = {
    "memory": plain.memory(4, 8, 16, 8.0),
    "memory, odd sizes": plain.memory(3, 5, 7, 2.0),
    "memory, tensor-core sizes": plain.memory(2, 64, 96, 12.0),
    "memory, keys of 128": plain.memory(2, 128, 64, 15.0),
    "pair": plain.pair(plain.attention(4, 2, 16, 0.25, conv=4, window=20, keep_first=2, rot=(16, 10000.0),
                                       scaling=(8.0, 1.0, 4.0, 32)),
                       plain.keep(2, 8, 16, (0.9, 0.99), rot=(8, 100.0))),
    "pair, no mask, part of odd heads rotated": plain.pair(plain.attention(3, 1, 20, 0.3, conv=2, rot=(6, 50.0)),
                                                           plain.keep(1, 6, 10, (0.97,), rot=(2, 10.0))),
    "pair at tensor-core sizes": plain.pair(
        plain.attention(8, 4, 64, 0.125, conv=3, window=36, keep_first=5, rot=(32, 10000.0)),
        plain.keep(3, 64, 32, (0.9, 0.98, 0.999), rot=(64, 10000.0))),
    "pair, heads of 128, all kept": plain.pair(
        plain.attention(4, 4, 128, 0.09, conv=1, window=9, keep_first=200, rot=(64, 500.0)),
        plain.keep(2, 128, 128, (0.95, 1.0), rot=(128, 10000.0))),
    "pair, neither convolution nor rotation": plain.pair(plain.attention(2, 2, 16, 0.25, window=3, keep_first=40),
                                                         plain.keep(2, 16, 8, (0.0, 0.5))),
}


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("what", list(ALONE))
def test_each_mixer_alone(tmp_path, what, dtype):
    cfg = plain.model(64, 48, 1e-5, [(ALONE[what], None)], bigram=(17, 3, 5))
    d = str(tmp_path / "alone")
    cfg, w = write_model(d, cfg=cfg, seed=len(what), sharp=SHARP[dtype])
    reqs = requests_of(cfg, [1, 2, 19, 20, 21, 22, 47, 90, 140], 3)
    ref = {rid: plain.forward(cfg, w, t).numpy() for rid, t in reqs.items()}
    for steps in (helpers.trace_whole(reqs), helpers.trace_prefill_then_decode(reqs, tail=25),
                  helpers.trace_mixed(reqs, max_live=3, seed=2, portion_choices=(2, 3, 33, 9, 70))):
        eng = engine_of(d, dtype, 8, helpers.max_live_tokens(steps, round_to=64), max_requests=3)
        rows = helpers.replay(eng, steps)
        compare(rows, ref, dtype, f"{what} {dtype}")


# ---------------------------------------------------------------------------------------------
# GPU: whole models under every cutting
# ---------------------------------------------------------------------------------------------
# prompt lengths just below, at and just above the windows (21 and 33; 1; 36 and 5), the kept tokens (3 and 9; 17 and
# 1), and the pages' borders (8; 4; 16)
LENGTHS = {"A": [1, 2, 3, 4, 8, 9, 10, 21, 22, 24, 33, 34, 60, 97], "B": [1, 3, 4, 5, 8, 9, 31, 32, 75],
           "C": [2, 4, 5, 6, 7, 16, 17, 18, 36, 37, 53, 70, 130, 200]}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name in plain.CONFIGS:
        for dtype, sharp in SHARP.items():
            d = str(tmp_path_factory.mktemp("duz" + name))
            cfg, w = write_model(d, name, seed=ord(name), sharp=sharp)
            reqs = requests_of(cfg, LENGTHS[name], 2)
            ref = {rid: plain.forward(cfg, w, t).numpy() for rid, t in reqs.items()}
            out[name, dtype] = (d, cfg, w, reqs, ref, plain.CONFIGS[name][1])
    return out


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(plain.CONFIGS))
@pytest.mark.parametrize("mode", ["whole", "decode from the first token", "decode40", "portions", "mixed"])
def test_replay_matches_plain(models, name, dtype, mode):
    d, cfg, w, reqs, ref, page = models[name, dtype]
    if mode == "whole":
        steps = helpers.trace_whole(reqs)
    elif mode == "decode from the first token":
        steps = helpers.trace_prefill_then_decode(reqs, tail=10 ** 6)
    elif mode == "decode40":
        steps = helpers.trace_prefill_then_decode(reqs, tail=40)
    elif mode == "portions":
        steps = helpers.trace_portions(reqs)
    else:
        steps = helpers.trace_mixed(reqs, max_live=4, seed=5)
    pool = helpers.max_live_tokens(steps, round_to=max(64, page))
    eng = engine_of(d, dtype, page, pool, max_requests=4)
    rows = helpers.replay(eng, steps)
    assert len(rows) == sum(len(t) for t in reqs.values())
    worst = compare(rows, ref, dtype, f"{name} {dtype} {mode}")
    print(f"[worst] {name}, {dtype}, {mode}: {worst:.3e}")
    eng.cache.check_consistency()
    assert all(p.used_pages == 0 for p in eng.cache.pools)


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_portions_and_graphs(models, dtype):
    """Portions of more than 64 tokens after a cached prefix beside decode steps replayed from CUDA graphs."""
    d, cfg, w, reqs, ref, page = models["C", dtype]
    steps = helpers.trace_mixed(reqs, max_live=3, seed=13, prefill_frac=0.8, portion_choices=(70, 130, 65, 2, 100))
    pool = helpers.max_live_tokens(steps, round_to=64)
    eng = engine_of(d, dtype, page, pool, max_requests=4, use_graphs=True)
    rows = helpers.replay(eng, steps)
    worst = compare(rows, ref, dtype, f"C {dtype} long portions, graphs")
    print(f"[worst] C, {dtype}, long portions, graphs: {worst:.3e}")
    assert eng.graph_replays > 0


FUZZ_SEEDS = int(os.environ.get("CCB_FUZZ_SEEDS", "12"))


@gpu
@pytest.mark.parametrize("seed", range(FUZZ_SEEDS))
def test_random_configurations(tmp_path, seed):
    """Configurations drawn at random (sizes, head counts, the order of the layers, windows, kept tokens, taps,
    constants, with and without pair table, side input, rotation, scaling, mask and feed-forward): a mixed trace with a
    pool that is just large enough, and every request whole, in both types.  A drawn model has rows that magnify
    rounding (a side input of three columns is normalised whatever its size, a memory of four key channels may nearly
    cancel), so the 32-bit bound of a row grows with how far that row moves in the plain implementation when every
    weight is changed by a millionth; the bfloat16 runs, which are there for the kernels' paths at odd sizes, want
    finite rows, a median within 3e-2, and beyond 8e-2 at most one row in eight, or half as many again as the plain
    implementation moves that far when every weight is changed by half a bfloat16 step (choices of experts flip)."""
    cfg, page = plain.random_config(1000 + seed)
    d = str(tmp_path / "drawn")
    cfg, w = write_model(d, cfg=cfg, seed=seed, sharp=1.5)
    reqs = requests_of(cfg, [1, 2, page, page + 1, 35, 72, 74, 110], seed)
    ref = {rid: plain.forward(cfg, w, t).numpy() for rid, t in reqs.items()}
    gen = torch.Generator().manual_seed(seed)
    scale = {rid: max(1e-6, float(np.abs(r).max())) for rid, r in ref.items()}

    def moves(by):   # per request: how far each row moves when every weight is changed by that share
        moved = {k: v.double() * (1 + by * torch.randn(v.shape, dtype=torch.float64, generator=gen)) for k, v in w.items()}
        return {rid: np.abs(plain.forward(cfg, moved, t).numpy() - ref[rid]).max(1) / scale[rid] for rid, t in reqs.items()}

    bound = {rid: TOL32 + 10 * m for rid, m in moves(1e-6).items()}
    far_rows = sum(int((m > TOL16).sum()) for m in moves(2e-3).values())
    for dtype in ("float32", "bfloat16"):
        for steps in (helpers.trace_mixed(reqs, max_live=4, seed=seed, portion_choices=(2, 3, 5, 17, 40)),
                      helpers.trace_whole(reqs)):
            pool = helpers.max_live_tokens(steps, round_to=max(64, page))
            eng = engine_of(d, dtype, page, pool, max_requests=4, use_graphs=(dtype == "bfloat16"))
            rows = helpers.replay(eng, steps)
            if dtype == "float32":
                for (rid, pos), row in rows.items():
                    err = float(np.abs(row - ref[rid][pos]).max()) / scale[rid]
                    assert np.isfinite(row).all() and err <= bound[rid][pos], (seed, rid, pos, err, bound[rid][pos])
            else:
                errs = np.array([np.abs(row - ref[rid][pos]).max() / scale[rid] for (rid, pos), row in rows.items()])
                assert np.isfinite(errs).all() and np.median(errs) <= 3e-2, (seed, float(np.median(errs)))
                beyond = int((errs > TOL16).sum())
                assert beyond <= max(len(errs) // 8, 3 * far_rows // 2), (seed, beyond, far_rows, len(errs))
            assert all(p.used_pages == 0 for p in eng.cache.pools)


@gpu
def test_a_slot_that_is_used_again_starts_from_zero(models):
    """Two state slots, five requests one after another and in pairs: every later request gets a slot whose
    recurrent states, running maxima, convolution rows and previous token an earlier one left behind."""
    d, cfg, w, reqs, ref, page = models["A", "float32"]
    eng = engine_of(d, "float32", page, 256, max_requests=2)
    ids = list(reqs)[8:13]
    for group in ([ids[0]], [ids[1], ids[2]], [ids[3], ids[4]]):
        steps = helpers.trace_mixed({r: reqs[r] for r in group}, max_live=2, seed=1)
        rows = helpers.replay(eng, steps)
        helpers.compare(rows, ref, TOL32, "slots used again")
    assert eng.cache.slots.free_slots == 2


def _one_layer(mix, ff=None, **kw):
    return plain.model(64, 32, 1e-5, [(mix, ff)], **kw)


def _attention_decides(w, shared=(0, 1)):
    """A pair whose retention is switched off.  Queries and keys read the first half of the stream and the output the
    second: tokens 0 and 1 share their first half and have opposite second halves, so the query of token 1 matches the
    key of token 0 as well as its own and hardly any other; the value (which is the key) is read back through
    coordinates that carry the second half weakly."""
    p = "l0.mix."
    g = torch.Generator().manual_seed(3)
    base = torch.randn(16, 16, generator=g) / 4.0
    w[p + "left.k"] = torch.cat([base * 4.0, 0.15 * torch.randn(16, 16, generator=g)], 1)
    w[p + "left.q"] = torch.cat([torch.cat([base, base], 0) * 4.0, torch.zeros(32, 16)], 1)
    w[p + "left.q.norm"] = torch.ones_like(w[p + "left.q.norm"]) * 3.0
    w[p + "left.k.norm"] = torch.ones_like(w[p + "left.k.norm"]) * 3.0
    w[p + "right.out"] = torch.zeros_like(w[p + "right.out"])
    w["l0.norm1"], w["l0.norm1.b"] = torch.ones(32), torch.zeros(32)
    w["embed"][2:, :16] *= 0.2
    a, b = shared
    w["embed"][b, :16] = w["embed"][a, :16]
    w["embed"][b, 16:] = -w["embed"][a, 16:]


@gpu
@pytest.mark.parametrize("case", ["window", "kept"])
def test_a_key_at_an_edge_decides(tmp_path, case):
    """Attention over a window of 20 with two kept tokens.  Token 1 ends the sequence of 90.  "window": token 0 stands
    19 places back (the last key the window keeps) or 20 places back (the first it drops).  "kept": token 0 is the
    second token (the last that is kept) or the third.  In a prompt, in portions that end at the edge, and decoded, the
    pages between given back."""
    cfg = _one_layer(plain.pair(plain.attention(2, 1, 16, 0.25, conv=0, window=20, keep_first=2),
                                plain.keep(1, 8, 8, (0.9,))))
    d = str(tmp_path / "edge")
    cfg, w = write_model(d, cfg=cfg, seed=11, edit=_attention_decides)
    rng = np.random.RandomState(0)
    moves = {}
    for at in ((70, 69) if case == "window" else (1, 2)):
        toks = rng.randint(2, 64, size=90).tolist()
        toks[at], toks[-1] = 0, 1
        ref = plain.forward(cfg, w, toks).numpy()
        other = list(toks)
        other[at] = 2
        moves[at] = np.abs(ref[-1] - plain.forward(cfg, w, other).numpy()[-1]).max() / np.abs(ref[-1]).max()
        for dtype in ("float32", "bfloat16"):
            eng = engine_of(d, dtype, 8, 128)
            reqs = {"a": toks}
            for steps in (helpers.trace_whole(reqs), helpers.trace_prefill_then_decode(reqs, tail=40),
                          helpers.trace_portions(reqs, sizes=(at, 2, 10, 90 - at - 13, 1)),
                          helpers.trace_portions(reqs, sizes=(at + 1, 2, 86 - at, 1))):
                rows = helpers.replay(eng, steps)
                compare(rows, {"a": ref}, dtype, f"key at {at}")
    inside, outside = (70, 69) if case == "window" else (1, 2)
    assert moves[inside] > 0.05 and moves[outside] == 0.0, moves


@gpu
def test_the_one_in_the_denominator_decides(tmp_path):
    """Scores far below zero everywhere: nearly the whole of each softmax goes to the term without a key, and the
    attention's output (before its norm) all but vanishes; a plain softmax would give another direction."""
    cfg = _one_layer(plain.pair(plain.attention(3, 1, 16, 0.5, window=9, keep_first=1), plain.keep(1, 8, 8, (0.9,))))
    d = str(tmp_path / "one")

    def edit(w):   # every key the same direction, every query against it, by a token-dependent length
        p = "l0.mix.left."
        w[p + "k.norm"] = w[p + "k.norm"] * 1.5
        w[p + "q.norm"] = w[p + "q.norm"] * 1.5

    cfg, w = write_model(d, cfg=cfg, seed=12, edit=edit)
    toks = np.random.RandomState(1).randint(0, 64, size=40).tolist()
    ref = plain.forward(cfg, w, toks).numpy()
    kept = plain.softmax_plus_one
    try:
        plain.softmax_plus_one = lambda s, seen: torch.softmax(s.masked_fill(~seen, float("-inf")), -1)
        without = plain.forward(cfg, w, toks).numpy()
    finally:
        plain.softmax_plus_one = kept
    assert np.abs(without - ref).max() > 0.1 * np.abs(ref).max()
    for dtype in ("float32", "bfloat16"):
        eng = engine_of(d, dtype, 4, 64)
        for steps in (helpers.trace_whole({"a": toks}), helpers.trace_prefill_then_decode({"a": toks}, tail=20)):
            compare(helpers.replay(eng, steps), {"a": ref}, dtype, "one in the denominator")


@gpu
@pytest.mark.parametrize("which", ["memory", "retention"])
def test_a_far_token_decides_through_the_state(tmp_path, which):
    """One layer whose state keeps nearly everything.  q and k read the first half of the stream, v the second; tokens 0
    and 1 share their first half.  Token 0 stands at ONE far place among 400 and token 1 at the end: what the state kept
    of the far token decides the last logits.  The far place is the first token, around a page border and the middle;
    the prompt is cut so that the state crosses steps."""
    dk = 16
    if which == "memory":
        mix, p = plain.memory(2, dk, 16, 20.0), "l0.mix."
    else:
        mix, p = plain.pair(plain.attention(1, 1, 16, 0.25, window=2), plain.keep(2, dk, 16, (0.9999, 1.0))), "l0.mix.right."
    cfg = _one_layer(mix)
    d = str(tmp_path / "far")

    def edit(w):
        w[p + "v"][:, :16] = 0                        # v reads the second half
        w[p + "k"][:, 16:] = 0                        # k the first
        w[p + "k"] *= 2.0
        w[p + "q"] = w[p + "k"] * 1.0
        if which == "memory":
            w[p + "f"], w[p + "f.b"] = torch.zeros_like(w[p + "f"]), torch.full_like(w[p + "f.b"], 12.0)
            w[p + "i"], w[p + "i.b"] = torch.zeros_like(w[p + "i"]), torch.zeros_like(w[p + "i.b"])
        else:
            w["l0.mix.left.out"] = torch.zeros_like(w["l0.mix.left.out"])
        w["l0.norm1"], w["l0.norm1.b"] = torch.ones(32), torch.zeros(32)
        w["l0.norm1b"] = torch.full((32,), 3.0)       # the mixer outweighs the token's own row
        w["embed"][2:, :16] *= 0.05
        w["embed"][1, :16] = w["embed"][0, :16]

    cfg, w = write_model(d, cfg=cfg, seed=8, edit=edit)
    rng = np.random.RandomState(0)
    for far_at in (0, 7, 8, 200):
        toks = rng.randint(2, 64, size=400).tolist()
        toks[far_at], toks[-1] = 0, 1
        ref = plain.forward(cfg, w, toks).numpy()
        without = plain.forward(cfg, w, toks[:far_at] + [2] + toks[far_at + 1:]).numpy()
        assert np.abs(ref[-1] - without[-1]).max() > 0.1 * np.abs(ref[-1]).max()
        for dtype in ("float32", "bfloat16"):
            eng = engine_of(d, dtype, 8, 448)
            reqs = {"a": toks}
            for steps in (helpers.trace_whole(reqs), helpers.trace_prefill_then_decode(reqs, tail=3),
                          helpers.trace_portions(reqs, sizes=(150, 2, 100, 147, 1))):
                rows = helpers.replay(eng, steps)
                compare(rows, {"a": ref}, dtype, f"far token at {far_at}")


@gpu
def test_the_running_maximum_at_extreme_gates(tmp_path):
    """Input gates that jump between their caps and forget gates that drop everything or nothing: without the running
    maximum the exponentials of the sums would overflow a float."""
    cfg = _one_layer(plain.memory(3, 8, 8, 60.0), bigram=(19, 3, 5))
    d = str(tmp_path / "extreme")

    def edit(w):
        w["l0.mix.i"] = w["l0.mix.i"] * 120.0
        w["l0.mix.f"] = w["l0.mix.f"] * 40.0

    cfg, w = write_model(d, cfg=cfg, seed=3, edit=edit)
    reqs = requests_of(cfg, [1, 2, 33, 64, 65, 150], 7)
    ref = {rid: plain.forward(cfg, w, t).numpy() for rid, t in reqs.items()}
    for dtype in ("float32", "bfloat16"):
        for steps in (helpers.trace_whole(reqs), helpers.trace_portions(reqs), helpers.trace_mixed(reqs, max_live=3)):
            eng = engine_of(d, dtype, 8, 512)
            rows = helpers.replay(eng, steps)
            assert all(np.isfinite(r).all() for r in rows.values())
            if dtype == "float32":
                helpers.compare(rows, ref, 1e-3, "extreme gates")   # (gates of 60: their rounding is magnified 120-fold)


@gpu
def test_the_pair_table_decides_across_portions(tmp_path):
    """The tokens' own rows are nearly switched off, so the stream starts from the row that (previous token, token)
    chooses: a wrong previous token at the start of a portion, or the wrong row at position 0, changes every logit of
    that position."""
    cfg = _one_layer(plain.memory(2, 8, 8, 5.0), plain.dense(24), bigram=(29, 7, 11))
    d = str(tmp_path / "pairs")
    cfg, w = write_model(d, cfg=cfg, seed=5, edit=lambda w: w.update(embed=w["embed"] * 0.01))
    reqs = requests_of(cfg, [1, 2, 9, 30], 7)
    ref = {rid: plain.forward(cfg, w, t).numpy() for rid, t in reqs.items()}
    for dtype in ("float32", "bfloat16"):
        for steps in (helpers.trace_whole(reqs), helpers.trace_portions(reqs, sizes=(1, 2, 3, 1, 5)),
                      helpers.trace_mixed(reqs, max_live=2, seed=3, portion_choices=(2, 3))):
            eng = engine_of(d, dtype, 4, 128, max_requests=2)
            rows = helpers.replay(eng, steps)
            compare(rows, ref, dtype, "pair table")


@gpu
def test_long_decoding(models):
    """260 tokens one by one: the windows pass over decoded tokens many times, their pages are given back and the
    kept ones stay."""
    rng = np.random.RandomState(9)
    for dtype in ("float32", "bfloat16"):
        d, cfg, w, reqs, ref, page = models["A", dtype]
        toks = rng.randint(0, cfg["vocab"], size=260).tolist()
        want = plain.forward(cfg, w, toks).numpy()
        eng = engine_of(d, dtype, page, 320, use_graphs=(dtype == "bfloat16"))
        steps = helpers.trace_prefill_then_decode({"a": toks}, tail=10 ** 6)
        rows = helpers.replay(eng, steps)
        worst = compare(rows, {"a": want}, dtype, f"long decoding {dtype}")
        print(f"[worst] long decoding, {dtype}: {worst:.3e}")
        # a window of 33 with nine kept tokens over pages of 8: at most two kept pages and six of the window
        assert max(p.high_water for p in eng.cache.pools) <= 8


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(models, dtype):
    """Prompts of unequal length in portions of 7 through ``LLM.generate`` and its scheduler."""
    from ccinfer_b200 import LLM, SamplingParams
    d, cfg, w, reqs, ref, page = models["A", dtype]
    rng = np.random.RandomState(4)
    prompts = [rng.randint(0, cfg["vocab"], size=n).tolist() for n in (1, 9, 20, 33)]
    llm = LLM(d, dtype=dtype, page_size=page, kv_tokens=512, prefill_chunk_size=7, max_requests=4,
              max_tokens_per_step=64)
    got = llm.generate(prompts, SamplingParams(max_tokens=10))
    if dtype == "float32":
        assert got == [plain.greedy(cfg, w, p, 10) for p in prompts]
    else:   # rounding may flip an argmax between two close logits: every token must be (nearly) the best one
        for p, new in zip(prompts, got):
            toks = list(p)
            for t in new:
                row = plain.forward(cfg, w, toks)[-1]
                assert row[t] >= row.max() - 0.1 * row.abs().max()
                toks.append(t)
    assert all(pool.used_pages == 0 for pool in llm.engine.cache.pools)


@gpu
def test_a_preempted_request_starts_its_state_again(models):
    """So few pages that a request is preempted and computed again (its slot is closed and opened: the recurrent
    states, the running maxima and the previous token start again, the pages are taken anew): the greedy tokens are
    those of a calm run."""
    from ccinfer_b200 import LLM, SamplingParams
    d, cfg, w, reqs, ref, page = models["A", "float32"]
    rng = np.random.RandomState(6)
    prompts = [rng.randint(0, cfg["vocab"], size=n).tolist() for n in (20, 26, 17)]
    llm = LLM(d, dtype="float32", page_size=page, kv_tokens=8 * page, prefill_chunk_size=16, max_requests=4,
              max_tokens_per_step=64)
    got = llm.generate(prompts, [SamplingParams(max_tokens=n) for n in (24, 20, 28)])
    assert llm.scheduler.preemptions > 0
    assert got == [plain.greedy(cfg, w, p, n) for p, n in zip(prompts, (24, 20, 28))]
    llm.engine.cache.check_consistency()


@gpu
def test_the_programs_as_a_user_calls_them(models, tmp_path):
    """bin/ccinfer: greedy tokens of a model folder; a random model written from a configuration generates the
    same tokens as the same configuration drawn on the device; bin/trace_run: a mixed trace over four request
    slots, its files against the plain logits."""
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    d, cfg, w, reqs, ref, page = models["A", "float32"]
    exe = [sys.executable, os.path.join(root, "bin", "ccinfer")]
    prompt = list(reqs.values())[9]
    r = subprocess.run(exe + ["--model-path", d, "--dtype", "float32", "--page-size", str(page), "--kv-tokens", "256",
                              "--max-tokens", "6", "--prompt-ids", ",".join(map(str, prompt))],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert json.loads(r.stdout.strip().splitlines()[0])["token_ids"] == plain.greedy(cfg, w, prompt, 6)

    cj = str(tmp_path / "config.json")
    with open(cj, "w") as f:
        json.dump(cfg, f)
    common = ["--dtype", "float32", "--kv-tokens", "256", "--max-tokens", "5", "--random-prompts", "9,4",
              "--weights-seed", "5", "--weights-std", "0.3"]
    a = subprocess.run(exe + ["--random-config", cj] + common, capture_output=True, text=True, timeout=600)
    assert a.returncode == 0, a.stderr[-2000:]
    made = str(tmp_path / "made")
    wr = subprocess.run(exe + ["--model-path", made, "--write-random-model", cj, "--weights-seed", "5",
                               "--weights-std", "0.3"], capture_output=True, text=True, timeout=600)
    assert wr.returncode == 0, wr.stderr[-2000:]
    b = subprocess.run(exe + ["--model-path", made] + common, capture_output=True, text=True, timeout=600)
    assert b.returncode == 0, b.stderr[-2000:]
    assert a.stdout == b.stdout and len(a.stdout.strip().splitlines()) == 2

    steps = helpers.trace_mixed(reqs, max_live=4, seed=3)
    pool = helpers.max_live_tokens(steps)
    out_dir = tmp_path / "out"
    lines = "".join(json.dumps({"step": i, **st}) + "\n" for i, st in enumerate(steps))
    t = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out",
                        str(out_dir), "--max-tokens", str(pool)], input=lines, capture_output=True, text=True,
                       timeout=600)
    assert t.returncode == 0, t.stderr[-2000:]
    assert t.stdout.split() == [x for i in range(len(steps)) for x in ("done", str(i))]
    rows, seen = {}, {rid: 0 for rid in reqs}
    for i, st in enumerate(steps):
        n_want = sum(len(e["want"]) for e in st["entries"])
        arr = np.fromfile(out_dir / f"{i}.f32", dtype="<f4").reshape(n_want, cfg["vocab"])
        at = 0
        for e in st["entries"]:
            for wnt in e["want"]:
                rows[(e["id"], seen[e["id"]] + wnt)] = arr[at]
                at += 1
            seen[e["id"]] += len(e["tokens"])
    assert len(rows) == sum(len(x) for x in reqs.values())
    helpers.compare(rows, ref, TOL32, "trace_run")
