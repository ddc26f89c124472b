"""Toripel in the engine against the plain implementation of ``plain_toripel``.

Configuration, plan, shared caches and random tables on the CPU; on the GPU the kernels of the design alone, each mixer
and the mixture as parts of small models, then whole models under every way of cutting the work: whole prompts,
token-by-token decoding from the first token, portions down to two tokens, mixed batches with pages and state slots that
are used again; keys just inside and just outside a window, also of a layer that reads another one's rows through a
wider window; sinks; a far token that decides through the recurrent state and through the convolution's ring; the table's
experts of tokens that are still on the device; long decoding; greedy generation through the Python entry point and its
scheduler; the programs.
"""
import copy
import json
import math
import os

import numpy as np
import pytest
import torch

import helpers
import plain_toripel as plain

gpu = pytest.mark.gpu

TOL32 = 5e-5          # relative to the largest logit of the request
TOL16 = 3e-2
SHARP = {"float32": 3.0, "bfloat16": 1.5}   # the latent layers' queries times this: the softmax sits on few keys


def write_model(path, name=None, cfg=None, seed=0, sharp=1.0, edit=None):
    from safetensors.torch import save_file
    if cfg is None:
        cfg, _ = plain.config(name)
    w = plain.random_weights(cfg, seed, sharp)
    if edit is not None:
        edit(w)
        w = {k: v.to(torch.bfloat16).to(torch.float32) if v.is_floating_point() else v for k, v in w.items()}
    os.makedirs(path, exist_ok=True)
    save_file({k: (v.to(torch.bfloat16) if v.is_floating_point() else v).contiguous() for k, v in w.items()},
              os.path.join(path, "model.safetensors"))
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    return cfg, w


def engine_of(path, dtype, page, pool, max_requests=4, use_graphs=False, step_tokens=None):
    from ccinfer_b200.engine.engine import Engine, EngineOptions
    return Engine.from_model_dir(path, EngineOptions(
        dtype=dtype, page_size=page, kv_tokens=pool, max_requests=max_requests,
        max_tokens_per_step=step_tokens or pool, max_context=pool, use_graphs=use_graphs))


# by what share every weight is changed to see how a row is conditioned: a millionth, or half a bfloat16 step
NUDGE = {"float32": 1e-6, "bfloat16": 2e-3}


def bounds_of(cfg, w, reqs, ref, dtype, seed=0):
    """Per request the bound of each row's error: the type's tolerance, and ten times how far that row moves in the plain
    implementation when every weight is changed a little (a weighted sum of the copies, or a head's output before it is
    normed, may nearly cancel; a wrong mechanism moves rows by their own size)."""
    gen = torch.Generator().manual_seed(seed)
    moved = {k: v.double() * (1 + NUDGE[dtype] * torch.randn(v.shape, dtype=torch.float64, generator=gen))
             if v.is_floating_point() else v for k, v in w.items()}
    tol = TOL32 if dtype == "float32" else TOL16
    return {rid: tol + 10 * np.abs(plain.forward(cfg, moved, t).numpy() - ref[rid]).max(1) / max(1e-6, np.abs(ref[rid]).max())
            for rid, t in reqs.items()}


def compare(rows, ref, dtype, what, bounds=None):
    """The largest error, relative to the largest logit of the request, within the type's tolerance or each row's bound."""
    if bounds is None:
        return helpers.compare(rows, ref, TOL32 if dtype == "float32" else TOL16, what)
    worst = 0.0
    for (rid, pos), row in rows.items():
        err = float(np.abs(row - ref[rid][pos]).max()) / max(1e-6, float(np.abs(ref[rid]).max()))
        assert np.isfinite(row).all() and err <= bounds[rid][pos], (what, rid, pos, err, bounds[rid][pos])
        worst = max(worst, err)
    return worst


def requests_of(cfg, lengths, seed):
    rng = np.random.RandomState(seed)
    return {f"r{i}": rng.randint(0, cfg["vocab"], size=n).tolist() for i, n in enumerate(lengths)}


# ---------------------------------------------------------------------------------------------
# CPU: configuration, plan, caches read by other layers, random tables
# ---------------------------------------------------------------------------------------------
def test_config_is_read_written_and_refused():
    from ccinfer_b200.config.registry import architecture_of
    from ccinfer_b200.config.toripel import ToripelConfig
    from ccinfer_b200.errors import ModelConfigInvalid
    cfg, _ = plain.config("A")
    assert architecture_of(cfg).name == "Toripel"
    c = ToripelConfig.from_json(cfg)
    assert [l.type for l in c.layers] == ["latent_attention", "delta", "latent_attention", "attention", "latent_attention"]
    assert c.streams == 2 and c.embed_scale == 3.0 and c.layers[2].mlp is None
    m = c.layers[4].mixer
    assert (m.window, m.kv_from, m.q_rank, m.rot.scaling.fast) == (9, 0, 24, 8.0) and c.layers[1].mlp.top == 3
    for name in plain.CONFIGS:
        full = ToripelConfig.from_json(plain.config(name)[0])
        assert ToripelConfig.from_json(full.to_json()) == full
    b = ToripelConfig.from_json(plain.config("B")[0])
    assert b.layers[0].mixer.window is None and b.layers[1].mixer.rot.scaling is None
    for damage in (lambda j: j.pop("width"), lambda j: j.pop("streams"), lambda j: j.update(streams=0),
                   lambda j: j["norm"].pop("eps"), lambda j: j["norm"].update(eps=0.0), lambda j: j["embedding"].pop("scale"),
                   lambda j: j["layers"][0]["mixer"].pop("q_rank"), lambda j: j["layers"][0]["mixer"].pop("rot"),
                   lambda j: j["layers"][0]["mixer"]["rot"].update(dims=6),
                   lambda j: j["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"),
                   lambda j: j["layers"][0]["mixer"]["mask"].pop("size"),
                   lambda j: j["layers"][0]["mixer"]["mask"].update(size=0),
                   lambda j: j["layers"][2]["mixer"].update(kv_from=2), lambda j: j["layers"][2]["mixer"].update(kv_from=1),
                   lambda j: j["layers"][4]["mixer"].update(kv_from=2), lambda j: j["layers"][2]["mixer"].update(kv_rank=8),
                   lambda j: j["layers"][2]["mixer"]["rot"].update(base=5.0),
                   lambda j: j["layers"][1]["mixer"].pop("conv"), lambda j: j["layers"][1]["mixer"].update(kv_heads=3),
                   lambda j: j["layers"][3]["mixer"].update(kv_heads=3), lambda j: j["layers"][3]["mixer"].pop("vdim"),
                   lambda j: j["layers"][3].update(type="mamba2"), lambda j: j["layers"][0]["mlp"].pop("router"),
                   lambda j: j["layers"][0]["mlp"]["router"].update(top=6), lambda j: j["layers"][0]["mlp"].update(kind="dense"),
                   lambda j: j["layers"][0]["mlp"]["expert"].pop("ff"), lambda j: j["layers"][0].pop("mlp"),
                   lambda j: j.update(layers=[])):
        j = copy.deepcopy(cfg)
        damage(j)
        with pytest.raises(ModelConfigInvalid):
            ToripelConfig.from_json(j)


def test_plan_names_every_tensor_and_shares_the_latent_rows():
    from ccinfer_b200.architectures.toripel import build_plan
    from ccinfer_b200.config.toripel import ToripelConfig
    for cfg in [plain.config(n)[0] for n in plain.CONFIGS] + [plain.random_config(s)[0] for s in range(40)]:
        plan = build_plan(ToripelConfig.from_json(cfg))
        plan.validate()
        assert {s.name: tuple(s.shape) for s in plan.tensor_specs()} == plain.tensor_shapes(cfg)
    plan = build_plan(ToripelConfig.from_json(plain.config("A")[0]))
    assert [e.cache_of for e in plan.order] == [None, None, 0, None, 0]


def test_a_need_covers_the_layers_that_read_it():
    from ccinfer_b200.parts import CacheNeed
    kv = CacheNeed.keys_and_values
    assert kv(1, 8, window=24).covering(kv(1, 8, window=40)).window == 40
    assert kv(1, 8, window=24).covering(kv(1, 8, window=9)).window == 24
    assert kv(1, 8, window=24).covering(kv(1, 8)).group_key == ("all",)
    assert kv(1, 8).covering(kv(1, 8, window=3)).group_key == ("all",)
    assert kv(1, 8, chunk=8).covering(kv(1, 8, chunk=8)).group_key == ("chunk", 8)
    assert kv(1, 8, chunk=8).covering(kv(1, 8, window=8)).group_key == ("all",)
    both = kv(1, 8, window=24, keep_first=2).covering(kv(1, 8, window=9, keep_first=5))
    assert (both.window, both.keep_first) == (24, 5)


def test_random_tables_and_unit_matrices():
    """Rows of different numbers in range, every number drawn about equally often, the same for the same seed and name."""
    from ccinfer_b200.parts import TensorSpec
    from ccinfer_b200.weights.loader import random_tensor
    spec = TensorSpec("l0.mlp.table", (4000, 5), role="table", below=9)
    t = random_tensor(spec, 3, 0.02)
    assert t.dtype == torch.int32 and t.min() == 0 and t.max() == 8
    assert all(len(set(row)) == 5 for row in t.tolist())
    counts = torch.bincount(t.flatten().long(), minlength=9)
    assert (counts - 4000 * 5 / 9).abs().max() < 150
    assert torch.equal(t, random_tensor(spec, 3, 0.02)) and not torch.equal(t, random_tensor(spec, 4, 0.02))
    full = random_tensor(TensorSpec("t", (20, 7), role="table", below=7), 1, 0.02)
    assert torch.equal(full.sort(1).values, torch.arange(7, dtype=torch.int32).expand(20, 7))
    eye = random_tensor(TensorSpec("m", (4, 4), role="vector", init="eye_plus_normal"), 1, 0.01)
    assert (eye - torch.eye(4)).abs().max() < 0.1 and not torch.equal(eye, torch.eye(4))


def test_plain_connection_is_indexed_from_to():
    x = torch.tensor([[[1.0], [10.0]]], dtype=torch.float64)
    mix = torch.tensor([[0.0, 2.0], [0.0, 1.0]], dtype=torch.float64)       # both copies go to the second
    new = plain.write_streams(x, torch.tensor([[100.0]], dtype=torch.float64), mix, torch.tensor([1.0, 0.0]))
    assert new.flatten().tolist() == [100.0, 12.0]


def test_parts_refuse_what_they_do_not_compute():
    from ccinfer_b200.errors import Unsupported
    from ccinfer_b200.parts import (GroupedQueryAttention, HeadGatedDelta, HyperConnectionBlock, MixtureOfExperts, NoPosition,
                                    StreamsNorm)
    names = {"table": "t", "gate": "g{e}", "up": "u{e}", "down": "d{e}"}
    with pytest.raises(Unsupported):
        StreamsNorm(16, 17, 1e-5, "n")
    with pytest.raises(Unsupported):
        MixtureOfExperts(16, 4, 2, 8, dict(names, router="r"), activation="swiglu", table_vocab=9)
    with pytest.raises(Unsupported):
        MixtureOfExperts(16, 4, 2, 8, names, groups=2, activation="swiglu", table_vocab=9)
    with pytest.raises(Unsupported):
        HeadGatedDelta(16, 3, 2, 8, 8, 2, 1e-5, {})
    with pytest.raises(Unsupported):
        HeadGatedDelta(16, 2, 2, 300, 8, 2, 1e-5, {})
    with pytest.raises(ValueError):
        HyperConnectionBlock(None, None, None, norm2=object())
    a = GroupedQueryAttention(16, 2, 1, 72, NoPosition(), {"q": "q", "k": "k", "v": "v", "o": "o"}, value_dim=88,
                              tensor_core_heads=True)
    assert a.hd == 128 and GroupedQueryAttention.kernel_head_dim(40, 64, True) == 64
    assert GroupedQueryAttention.kernel_head_dim(130, 8, True) == 144


# ---------------------------------------------------------------------------------------------
# GPU: the kernels alone
# ---------------------------------------------------------------------------------------------
def _close(got, want, dtype, tol=2e-6):
    """Within rounding: of the float sums, and for bfloat16 results of one last rounding."""
    want = want.double()
    lim = tol * max(1.0, float(want.abs().max())) + (want.abs() * 2.0 ** -8 if dtype == torch.bfloat16 else 0.0)
    assert ((got.double().cpu() - want).abs() <= lim).all(), float((got.double().cpu() - want).abs().max())


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("S,D,T", [(1, 48, 3), (2, 77, 3), (3, 1000, 3), (4, 4096, 3), (7, 520, 3), (16, 2048, 3), (4, 6000, 3),
                                   (2, 9000, 3), (1, 4096, 200), (2, 512, 200), (3, 77, 200), (3, 700, 200), (4, 2048, 200),
                                   (4, 4096, 70), (5, 640, 200), (16, 100, 200), (2, 8192, 90)])
def test_streams_step_kernel(dtype, S, D, T):
    """A mix of the copies, an output or experts' rows added, and the norm of a weighted sum: from equal copies, in place,
    rows by index, without an output, and the plain sum."""
    from ccinfer_b200 import kernels
    g = torch.Generator().manual_seed(S * D + T)
    x = torch.randn(T, S, D, generator=g)
    mix, out, win = torch.randn(S, S, generator=g), torch.randn(S, generator=g), torch.randn(S, generator=g) + 1.5
    w = 1 + 0.3 * torch.randn(D, generator=g)
    delta = torch.randn(T, D, generator=g).to(dtype)
    top = 3
    rows = torch.randn(T * top, D, generator=g)
    pos = torch.randperm(T * top, generator=g).to(torch.int32)
    pos[1] = -1                                                       # a choice that was left out
    eps = 1e-5

    def normed(new, weights=None):
        u = (new * (weights if weights is not None else torch.ones(S)).double()[None, :, None]).sum(1)
        return plain.rms_unit(u, eps) * w.double()

    def mixed(x, d):
        return plain.write_streams(x.double(), d.double(), mix.double(), out.double())

    cu = lambda t: t.cuda().contiguous()
    y = torch.empty(T, D, dtype=dtype, device="cuda")
    common = dict(w=cu(w), eps=eps, mix=cu(mix), weights_out=cu(out))
    # in place
    xd = cu(x)
    kernels.streams_step(y, xd, S, weights_in=cu(win), delta=cu(delta), x_out=xd, **common)
    new = mixed(x, delta)
    _close(xd, new, torch.float32)
    _close(y, normed(new, win), dtype, 1e-5)
    # experts' rows, nothing written back, rows by index, the plain sum
    picked = torch.stack([rows[p] if p >= 0 else torch.zeros(D) for p in pos.tolist()]).view(T, top, D).sum(1)
    idx = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32)
    xd, st = cu(x), torch.zeros(1, dtype=torch.int32, device="cuda")
    kernels.streams_step(y, xd, S, pairs=(cu(rows), cu(pos), top), row_idx=cu(idx), status=st, **common)
    _close(y[:3], normed(mixed(x, picked))[idx.long()], dtype, 1e-5)
    assert torch.equal(xd.cpu(), x) and int(st) == 0
    # equal copies, written out for the first time
    h = cu(x[:, 0])
    xo = torch.full((T, S, D), float("nan"), device="cuda")
    kernels.streams_step(y, h, S, weights_in=cu(win), delta=cu(delta), x_out=xo, **common)
    new = mixed(x[:, :1].expand(T, S, D), delta)
    _close(xo, new, torch.float32)
    _close(y, normed(new, win), dtype, 1e-5)
    # no output yet: the norm alone
    kernels.streams_step(y, cu(x), S, w=cu(w), eps=eps, weights_in=cu(win))
    _close(y, normed(x.double(), win), dtype, 1e-5)
    # a bad row is reported and gives zeros
    kernels.streams_step(y, cu(x), S, w=cu(w), eps=eps, row_idx=cu(torch.tensor([0, T], dtype=torch.int32)), status=st)
    assert int(st) == kernels.ST_BAD_ROW and float(y[1].abs().max()) == 0.0
    _close(y[:1], normed(x.double())[:1], dtype, 1e-5)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D", [48, 77, 4096])
def test_streams_step_from_the_embedding(dtype, D):
    from ccinfer_b200 import kernels
    g = torch.Generator().manual_seed(D)
    table = torch.randn(31, D, generator=g).to(dtype)
    ids = torch.tensor([3, 30, -2, 0], dtype=torch.int32)             # -2: the token of request slot 1
    pending = torch.tensor([9, 12], dtype=torch.int32)
    w, win = 1 + 0.3 * torch.randn(D, generator=g), torch.tensor([0.2, -0.9, 1.1])
    h, y = torch.empty(4, D, device="cuda"), torch.empty(4, D, dtype=dtype, device="cuda")
    st = torch.zeros(1, dtype=torch.int32, device="cuda")
    kernels.streams_step(y, None, 3, w=w.cuda(), eps=1e-5, weights_in=win.cuda(), x_out=h, table=table.cuda(), ids=ids.cuda(),
                         scale=1.7, pending=pending.cuda(), status=st)
    e = table[[3, 30, 12, 0]].double() * 1.7
    _close(h, e, torch.float32)
    _close(y, plain.rms_unit(e * float(win.sum()), 1e-5) * w.double(), dtype, 1e-5)
    assert int(st) == 0
    kernels.streams_step(y, None, 3, w=w.cuda(), eps=1e-5, x_out=h, table=table.cuda(), ids=torch.tensor([3, 31, 1, 0],
                         dtype=torch.int32, device="cuda"), scale=1.7, status=st)
    assert int(st) == kernels.ST_BAD_TOKEN and float(h[1].abs().max()) == 0.0


@gpu
@pytest.mark.parametrize("rows,E,top,BM", [(1, 3, 3, 16), (7, 16, 2, 16), (40, 5, 1, 16), (300, 9, 4, 128), (3000, 32, 4, 128)])
def test_table_of_experts_kernels(rows, E, top, BM):
    from ccinfer_b200 import kernels
    g = torch.Generator().manual_seed(rows)
    V = 50
    table = torch.rand((V, E), generator=g).argsort(1)[:, :top].to(torch.int32).contiguous()
    real = torch.randint(0, V, (rows,), generator=g)
    ids = real.to(torch.int32).clone()
    pending = torch.tensor([int(real[0]), 7], dtype=torch.int32)
    ids[0] = -1                                                        # still on the device
    eot = torch.zeros(rows, dtype=torch.int32)
    if rows > 2:
        eot[rows - 1] = -1                                             # padding of a replayed step
    chosen = [table[int(t)].tolist() if e >= 0 else [] for t, e in zip(real, eot)]
    ex = kernels.ExpertTable(table.cuda(), ids.cuda(), eot.cuda(), pending.cuda())
    st = torch.zeros(1, dtype=torch.int32, device="cuda")
    dense = torch.full((rows, E), float("nan"), device="cuda")
    kernels.moe_table_route(ex, dense, status=st)
    want = torch.zeros(rows, E)
    for t, c in enumerate(chosen):
        want[t, c] = 1.0 / top
    assert torch.equal(dense.cpu(), want) and int(st) == 0
    pairs = rows * top
    n_tiles = kernels.moe_max_tiles(pairs, E, BM)
    mk = lambda n, dt=torch.int32: torch.full((n,), 12345, dtype=dt, device="cuda")
    src, pp, rw = mk(pairs), mk(pairs), mk(pairs, torch.float32)
    tiles = [mk(n_tiles) for _ in range(3)]
    kernels.moe_table_sort(ex, E, BM, src, rw, pp, *tiles, status=st)
    src, pp, rw, (te, tr, tn) = src.cpu(), pp.cpu().view(rows, top), rw.cpu(), [t.cpu() for t in tiles]
    held = sorted(int(p) for p in pp.flatten() if p >= 0)
    assert held == list(range(sum(len(c) for c in chosen))) and int(st) == 0
    expert_of_row = {}
    for t, c in enumerate(chosen):
        for k in range(top):
            if not c:
                assert int(pp[t, k]) == -1
                continue
            p = int(pp[t, k])
            assert int(src[p]) == t and abs(float(rw[p]) - 1.0 / top) < 1e-7
            expert_of_row[p] = c[k]
    covered = []
    for e, r0, n in zip(te.tolist(), tr.tolist(), tn.tolist()):
        for p in range(r0, r0 + n):
            assert expert_of_row[p] == e
            covered.append(p)
        assert n <= BM
    assert sorted(covered) == held
    assert (src[len(held):] == 0).all()                                # the places of the pairs that were left out
    bad = table.clone()
    bad[int(real[0]), 0] = E
    kernels.moe_table_route(kernels.ExpertTable(bad.cuda(), ids.cuda(), eot.cuda(), pending.cuda()), dense, status=st)
    assert int(st) == kernels.ST_BAD_TOKEN


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T", [2, 100])
def test_latent_rows_kernel(dtype, T):
    """The cache row, the rotated query parts and the second latent vector's norm, together and each alone."""
    from ccinfer_b200 import kernels
    g = torch.Generator().manual_seed(T)
    H, d, r, R, N, rd = 3, 5, 6, 20, 11, 4
    amp, eps = 1.3, 1e-5
    proj = torch.randn(T, 64, generator=g).to(dtype)
    q = torch.randn(T, 40, generator=g).to(dtype)
    w, wn, f = 1 + 0.2 * torch.randn(R, generator=g), 1 + 0.2 * torch.randn(N, generator=g), torch.tensor([1.0, 0.3])
    pos = torch.randint(0, 50, (T,), generator=g).to(torch.int32)
    slot = torch.randperm(T + 3, generator=g)[:T].to(torch.int32)
    slot[0] = -1

    def rot(x):   # [T, ..., r]
        a = pos.double().view(T, *([1] * (x.dim() - 2)), 1) * f.double()
        cs, sn = torch.cos(a) * amp, torch.sin(a) * amp
        u, v = x[..., :2].double(), x[..., 2:4].double()
        return torch.cat([u * cs - v * sn, v * cs + u * sn, x[..., 4:].double()], -1)

    cache = torch.zeros(1, T + 3, R + r, dtype=dtype, device="cuda")
    qa = torch.zeros(T, H, R + r, device="cuda")
    cq = torch.full((T, 16), 9.0, dtype=dtype, device="cuda")
    on, oc = 8, 30
    args = (oc, w.cuda(), f.cuda(), rd, pos.cuda())
    tail = (H, d, r, R, eps)
    pd = proj.cuda()
    kernels.latent_prepare(pd, *args, slot.cuda(), cache, *tail, amp=amp, low=(on, N, wn.cuda(), cq))
    kernels.latent_prepare(q.cuda(), *args, None, None, *tail, q=q.cuda(), qa=qa, amp=amp)
    rows = torch.cat([plain.rms_unit(proj[:, oc:oc + R].double(), eps) * w.double(), rot(proj[:, oc + R:oc + R + r])], 1)
    for t in range(1, T):
        _close(cache[0, int(slot[t])], rows[t], dtype, 1e-5)
    assert sum(float(cache[0, s].abs().max()) > 0 for s in range(T + 3)) == T - 1
    _close(cq, torch.cat([plain.rms_unit(proj[:, on:on + N].double(), eps) * wn.double(), torch.zeros(T, 16 - N)], 1), dtype, 1e-5)
    qr = rot(q[:, :H * (d + r)].view(T, H, d + r)[..., d:])
    _close(qa[:, :, R:], qr, torch.float32, 1e-5)
    # all three in one launch
    both = torch.cat([proj, q], 1).cuda()
    c2, qa2, cq2 = torch.zeros_like(cache), torch.zeros_like(qa), torch.zeros_like(cq)
    kernels.latent_prepare(both, *args, slot.cuda(), c2, *tail, q=both[:, 64:], qa=qa2, amp=amp, low=(on, N, wn.cuda(), cq2))
    assert torch.equal(c2, cache) and torch.equal(qa2, qa) and torch.equal(cq2, cq)


def _delta_rows(proj, off, conv_w, A_log, dt_bias, G, H, dk, dv, hist):
    """float64 q, k, v, decay, beta of one request's rows, ``hist`` [n, C] the rows before them."""
    oq, ok, ov, ob, oa, _ = off
    p = proj.double()
    C = 2 * G * dk + H * dv
    x = torch.cat([p[:, oq:oq + G * dk], p[:, ok:ok + G * dk], p[:, ov:ov + H * dv]], 1)
    full = torch.cat([hist.double(), x], 0)
    y = plain.silu(plain.causal_conv(full, conv_w.double().t()))[hist.shape[0]:]
    T = x.shape[0]
    q, k, v = y[:, :G * dk].view(T, G, dk), y[:, G * dk:2 * G * dk].view(T, G, dk), y[:, 2 * G * dk:C].view(T, H, dv)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * dk ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    g = torch.exp(-torch.exp(A_log.double()) * plain.softplus(p[:, oa:oa + H] + dt_bias.double()))
    return q, k, v, g, torch.sigmoid(p[:, ob:ob + H]), full


def _delta_walk(q, k, v, g, b, S):
    """o [T, H, dv] and the state after, from S [H, dv, dk]."""
    T, H, dv = v.shape
    group = [h // (H // q.shape[1]) for h in range(H)]
    o = torch.zeros(T, H, dv, dtype=torch.float64)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = b[t][:, None] * (v[t] - torch.einsum("hvd,hd->hv", S, k[t, group]))
        S = S + u[:, :, None] * k[t, group][:, None, :]
        o[t] = torch.einsum("hvd,hd->hv", S, q[t, group])
    return o, S


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("G,H,dk,dv,taps", [(2, 4, 16, 24, 4), (1, 1, 7, 5, 3), (1, 2, 128, 128, 2), (3, 3, 64, 300, 1),
                                            (1, 3, 160, 20, 4), (2, 2, 32, 36, 6), (1, 8, 12, 12, 3)])
def test_delta_with_a_decay_per_head(dtype, G, H, dk, dv, taps):
    """Three requests in shuffled slots: portions, then single tokens beside another portion, then single tokens, the
    state and the convolution's ring handed from one kernel to the others, against a float64 walk."""
    from ccinfer_b200 import kernels
    g = torch.Generator().manual_seed(dk * taps)
    C = 2 * G * dk + H * dv
    pad = lambda n: -(-n // 8) * 8
    oq, ok, ov = 0, pad(G * dk), 2 * pad(G * dk)
    og = ov + pad(H * dv)
    off = (oq, ok, ov, og + pad(H * dv), og + pad(H * dv) + pad(H), og)
    width = off[4] + pad(H)
    conv_w = torch.randn(taps, C, generator=g) / math.sqrt(taps)
    A_log, dt_bias, w = 0.5 * torch.randn(H, generator=g), 0.5 * torch.randn(H, generator=g), 1 + 0.2 * torch.randn(dv, generator=g)
    rule = kernels.HeadDelta(off, conv_w.cuda(), A_log.cuda(), dt_bias.cuda(), G, H, dk, dv, dk ** -0.5, 1e-6)
    n_slots, slots = 5, [3, 0, 4]
    ring = torch.full((n_slots, taps, C), float("nan"), dtype=dtype, device="cuda")   # (never read before it is written)
    state = torch.zeros(n_slots, H, dv, dk, device="cuda")
    hist = [torch.zeros(0, C) for _ in slots]
    S = [torch.zeros(H, dv, dk, dtype=torch.float64) for _ in slots]
    eps = 1e-5
    tol = 2e-5 if dtype == torch.float32 else 2e-3
    # (tokens of each request; the step's order of entries: single tokens first)
    for counts in ((1, 2, 9), (1, 1, 3), (1, 1, 1), (1, 21, 2), (1, 1, 1), (1, 1, 1), (2, 3, 40), (1, 1, 1)):
        order = sorted(range(3), key=lambda i: counts[i] != 1)
        n1 = sum(c == 1 for c in counts)
        rows = [torch.randn(counts[i], width, generator=g).to(dtype) for i in order]
        proj = torch.cat(rows).cuda()
        T = proj.shape[0]
        cu = torch.tensor([0] + list(np.cumsum([counts[i] for i in order])), dtype=torch.int32).cuda()
        eot = torch.tensor([e for e, i in enumerate(order) for _ in range(counts[i])], dtype=torch.int32).cuda()
        pos = torch.tensor([hist[i].shape[0] + j for i in order for j in range(counts[i])], dtype=torch.int32).cuda()
        slot = torch.tensor([slots[i] for i in order], dtype=torch.int32).cuda()
        y = torch.full((T, H * dv), float("nan"), dtype=dtype, device="cuda")
        if n1:
            kernels.delta_head_step(rule, proj, ring, state, w.cuda(), eps, pos, cu, slot, y, n1)
        if n1 < 3:
            f = lambda *s: torch.full((T, *s), float("nan"), device="cuda")
            qn, kn, vv, gg, bb, o = f(G, dk), f(G, dk), f(H, dv), f(H), f(H), f(H, dv)
            kernels.delta_head_prepare(rule, proj, ring, pos, eot, cu, slot, qn, kn, vv, gg, bb, n1, T - n1)
            kernels.conv_ring_write(rule, proj, ring, pos, cu, slot, n1, 3 - n1)
            kernels.delta_head_recurrence(qn, kn, vv, gg, bb, state, o, cu, slot, n1, 3 - n1, G, H, dk, dv)
            kernels.gated_head_rmsnorm(y[n1:], o[n1:], proj[n1:, og:og + H * dv], w.cuda(), H, dv, eps, silu_gate=True)
        at = 0
        for e, i in enumerate(order):
            q, k, v, gd, b, full = _delta_rows(rows[e], off, conv_w, A_log, dt_bias, G, H, dk, dv, hist[i])
            want, S[i] = _delta_walk(q, k, v, gd, b, S[i])
            want = plain.rms_unit(want, eps) * w.double()
            want = want.reshape(counts[i], H * dv) * plain.silu(rows[e][:, og:og + H * dv].double())
            got = y[at:at + counts[i]].double().cpu()
            lim = tol * max(1.0, float(want.abs().max())) + (want.abs() * 2.0 ** -8 if dtype == torch.bfloat16 else 0.0)
            assert ((got - want).abs() <= lim).all(), (counts, i, float((got - want).abs().max()))
            assert (state[slots[i]].double().cpu() - S[i]).abs().max() < tol * max(1.0, float(S[i].abs().max()))
            hist[i] = full.to(dtype).float()
            at += counts[i]
    assert float(state[1].abs().max()) == float(state[2].abs().max()) == 0.0    # nobody else's slot


# ---------------------------------------------------------------------------------------------
# GPU: the mixture as a part, and each mixer as the only layer of a model
# ---------------------------------------------------------------------------------------------
@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,top,F,sparse", [(6, 2, 32, False), (6, 2, 32, True), (16, 1, 64, True), (5, 5, 24, True),
                                            (16, 1, 64, False), (3, 2, 11, False), (1, 1, 16, True)])
def test_experts_named_by_a_table(tmp_path, dtype, n, top, F, sparse, monkeypatch):
    """Every expert on every token or only the named ones (tiles of 16 rows and, in bfloat16 from some rows an expert on,
    tcgen05 tiles), the experts' rows added up by the sum into the copies; with graphs, whose padded rows have no
    experts."""
    from ccinfer_b200.parts import MixtureOfExperts
    if sparse:
        monkeypatch.setattr(MixtureOfExperts, "SPARSE_MIN_WEIGHTS", 1)
    cfg = plain.model(60, 64, 3, 1e-5, [(plain.attend(2, 1, 8, 8, 0.4, window=5), plain.moe(n, top, F)),
                                        (plain.delta(1, 1, 8, 8, 2), plain.moe(n, top, F))])
    d = str(tmp_path / "moe")
    cfg, w = write_model(d, cfg=cfg, seed=n + top)
    reqs = requests_of(cfg, [1, 5, 40, 150], 1)
    ref = {rid: plain.forward(cfg, w, t).numpy() for rid, t in reqs.items()}
    bounds = bounds_of(cfg, w, reqs, ref, dtype)
    for steps in (helpers.trace_whole(reqs), helpers.trace_mixed(reqs, max_live=3, seed=2),
                  helpers.trace_many_decoders({k: reqs[k] for k in ("r1", "r2", "r3")})):
        eng = engine_of(d, dtype, 8, helpers.max_live_tokens(steps, round_to=64), use_graphs=True)
        assert eng.plan.layers[0].ffn.use_sparse == (sparse and (dtype == "float32" or F % 8 == 0))
        compare(helpers.replay(eng, steps), ref, dtype, f"experts {n} {top} {F} {dtype}", bounds)
    assert eng.graph_replays > 0


ALONE = {
    "attention": plain.attend(4, 2, 16, 24, 0.5, window=20),
    "attention, no mask, odd sizes": plain.attend(3, 1, 10, 7, 0.6),
    "attention laid out in 128": plain.attend(6, 3, 96, 72, 0.15, window=21),
    "attention, heads above 128": plain.attend(2, 1, 136, 40, 0.1, window=47),
    "attention, a window of one": plain.attend(2, 2, 64, 64, 0.3, window=1),
    "latent": plain.latent(3, 8, 4, 12, 16, 20, 0.4, window=20, scaling=(4.0, 16, 4.0, 1.0)),
    "latent, odd sizes, no mask": plain.latent(2, 5, 2, 3, 13, 7, 0.5, base=100.0),
    "latent at tensor-core sizes": plain.latent(5, 16, 16, 40, 64, 72, 0.2, window=21, scaling=(8.0, 64, 32.0, 1.0)),
    "latent, many heads, a window of one": plain.latent(20, 8, 16, 8, 16, 16, 0.3, window=1),
    "delta": plain.delta(4, 2, 8, 16, 4),
    "delta, odd sizes": plain.delta(3, 1, 5, 7, 3),
    "delta, one tap": plain.delta(2, 2, 64, 36, 1),
    "delta, many taps": plain.delta(2, 1, 16, 8, 7),
    "delta, keys of 128": plain.delta(2, 1, 128, 136, 4),
}


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("what", list(ALONE))
def test_each_mixer_alone(tmp_path, what, dtype):
    cfg = plain.model(64, 48, 2, 1e-5, [(ALONE[what], None)])
    d = str(tmp_path / "alone")
    cfg, w = write_model(d, cfg=cfg, seed=len(what), sharp=SHARP[dtype])
    reqs = requests_of(cfg, [1, 2, 19, 20, 21, 22, 47, 90, 140], 3)
    ref = {rid: plain.forward(cfg, w, t).numpy() for rid, t in reqs.items()}
    bounds = bounds_of(cfg, w, reqs, ref, dtype)
    for steps in (helpers.trace_whole(reqs), helpers.trace_prefill_then_decode(reqs, tail=25),
                  helpers.trace_mixed(reqs, max_live=3, seed=2, portion_choices=(2, 3, 33, 9, 70))):
        eng = engine_of(d, dtype, 8, helpers.max_live_tokens(steps, round_to=64), max_requests=3)
        compare(helpers.replay(eng, steps), ref, dtype, f"{what} {dtype}", bounds)


# ---------------------------------------------------------------------------------------------
# GPU: whole models under every cutting
# ---------------------------------------------------------------------------------------------
# prompt lengths just below, at and just above the windows (24, 40, 9 and 17; none; 36, 33, 70 and 100; 1 and 20) and the
# pages' borders (8; 4; 16)
LENGTHS = {"A": [1, 2, 8, 9, 10, 16, 17, 18, 24, 25, 26, 39, 40, 41, 60, 97], "B": [1, 3, 4, 5, 8, 9, 31, 32, 75],
           "C": [2, 15, 16, 17, 33, 34, 36, 37, 70, 71, 100, 101, 130, 200], "D": [1, 2, 15, 16, 17, 19, 20, 21, 22, 70]}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name in plain.CONFIGS:
        for dtype, sharp in SHARP.items():
            d = str(tmp_path_factory.mktemp("tor" + name))
            cfg, w = write_model(d, name, seed=ord(name), sharp=sharp)
            reqs = requests_of(cfg, LENGTHS[name], 2)
            ref = {rid: plain.forward(cfg, w, t).numpy() for rid, t in reqs.items()}
            out[name, dtype] = (d, cfg, w, reqs, ref, plain.CONFIGS[name][1])
            out["bounds", name, dtype] = bounds_of(cfg, w, reqs, ref, dtype)
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
    worst = compare(rows, ref, dtype, f"{name} {dtype} {mode}", models["bounds", name, dtype])
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
    worst = compare(rows, ref, dtype, f"C {dtype} long portions, graphs", models["bounds", "C", dtype])
    print(f"[worst] C, {dtype}, long portions, graphs: {worst:.3e}")
    assert eng.graph_replays > 0


FUZZ_SEEDS = int(os.environ.get("CCB_FUZZ_SEEDS", "16"))


@gpu
@pytest.mark.parametrize("seed", range(FUZZ_SEEDS))
def test_random_configurations(tmp_path, seed):
    """Configurations drawn at random (sizes, head counts, the order of the layers, windows, taps, copies, constants, with
    and without scaling, mask and feed-forward, layers that read others' rows): a mixed trace with a pool that is just
    large enough, and every request whole, in both types."""
    cfg, page = plain.random_config(1000 + seed)
    d = str(tmp_path / "drawn")
    cfg, w = write_model(d, cfg=cfg, seed=seed, sharp=1.5)
    reqs = requests_of(cfg, [1, 2, page, page + 1, 35, 72, 74, 110], seed)
    ref = {rid: plain.forward(cfg, w, t).numpy() for rid, t in reqs.items()}
    for dtype in ("float32", "bfloat16"):
        bounds = bounds_of(cfg, w, reqs, ref, dtype)
        for steps in (helpers.trace_mixed(reqs, max_live=4, seed=seed, portion_choices=(2, 3, 5, 17, 40)),
                      helpers.trace_whole(reqs)):
            pool = helpers.max_live_tokens(steps, round_to=max(64, page))
            eng = engine_of(d, dtype, page, pool, max_requests=4, use_graphs=(dtype == "bfloat16"))
            worst = compare(helpers.replay(eng, steps), ref, dtype, f"drawn configuration {seed}", bounds)
            print(f"[worst] drawn {seed}, {dtype}: {worst:.3e}")
            assert all(p.used_pages == 0 for p in eng.cache.pools)


@gpu
def test_a_slot_that_is_used_again_starts_from_zero(models):
    """Two state slots, five requests one after another and in pairs: every later request gets a slot whose recurrent
    states and convolution ring an earlier one left behind."""
    d, cfg, w, reqs, ref, page = models["A", "float32"]
    eng = engine_of(d, "float32", page, 256, max_requests=2)
    ids = list(reqs)[9:14]
    for group in ([ids[0]], [ids[1], ids[2]], [ids[3], ids[4]]):
        steps = helpers.trace_mixed({r: reqs[r] for r in group}, max_live=2, seed=1)
        rows = helpers.replay(eng, steps)
        helpers.compare(rows, ref, TOL32, "slots used again")
    assert eng.cache.slots.free_slots == 2


def _one_layer(*mixes, vocab=64):
    """Layers without feed-forwards over one copy of a stream of 32."""
    return plain.model(vocab, 32, 1, 1e-5, [(m, None) for m in mixes])


def _plain_stream(w, p):
    """The layer's connection as an ordinary residual sum, its norm without a weight."""
    w[p + "hc1.in"], w[p + "hc1.out"], w[p + "hc1.mix"] = torch.ones(1), torch.ones(1), torch.ones(1, 1)
    w[p + "norm1"] = torch.zeros(32)


def _twins(w):
    """Tokens 0 and 1 share the first half of their rows and have opposite second halves; the others' first halves are
    small."""
    w["embed"][2:, :16] *= 0.2
    w["embed"][1, :16] = w["embed"][0, :16]
    w["embed"][1, 16:] = -w["embed"][0, 16:]


def _edge_attention(w, p):
    """Queries and keys read the first half of the stream alike, values the second."""
    w[p + "k"][:, 16:] = 0
    w[p + "v"][:, :16] = 0
    w[p + "q"] = torch.cat([w[p + "k"], w[p + "k"]], 0)
    for b in ("q.b", "k.b", "v.b"):
        w[p + b] = torch.zeros_like(w[p + b])


def _edge_latent(w, p, own=True):
    """The latent vector is [16 coordinates of the first half | 16 of the second]; queries and keys read the first 16,
    values the last; no rotated part to speak of, a sink far below."""
    eye = torch.eye(32)
    if own:
        w[p + "dkv"] = torch.cat([eye * 1.0, torch.zeros(2, 32)], 0)
        w[p + "dkv.norm"] = torch.ones(32)
    w[p + "dq"], w[p + "dq.norm"] = eye.clone(), torch.ones(32)
    key = torch.cat([eye[:16], torch.zeros(0, 32)], 0)
    w[p + "uk"] = key.clone()
    w[p + "uq"] = torch.cat([key * 4.0, torch.zeros(2, 32)], 0)
    w[p + "uv"] = torch.cat([torch.zeros(16, 16), torch.eye(16)], 1)
    w[p + "sink"] = torch.full((1,), -20.0)
    w[p + "o"] = 2.0 * torch.randn(32, 16, generator=torch.Generator().manual_seed(4))


EDGES = {
    # (layers, the layer whose window decides, the window)
    "attention": ([plain.attend(2, 1, 16, 16, 8.0, window=20)], 20),
    "latent": ([plain.latent(1, 16, 2, 16, 32, 32, 0.5, window=20)], 20),
    # the layer that owns the rows sees 5 of them, the one that reads them 20: the rows must outlive the owner's window
    "latent rows read through a wider window": ([plain.latent(1, 16, 2, 16, 32, 32, 0.5, window=5),
                                                 plain.latent(1, 16, 2, 16, 32, 32, 0.5, window=20, kv_from=0)], 20),
    "latent rows read through a narrower window": ([plain.latent(1, 16, 2, 16, 32, 32, 0.5, window=70),
                                                    plain.latent(1, 16, 2, 16, 32, 32, 0.5, window=20, kv_from=0)], 20),
}


@gpu
@pytest.mark.parametrize("case", list(EDGES))
def test_a_key_at_the_windows_edge_decides(tmp_path, case):
    """Tokens 0 and 1 share what queries and keys read, so the query of token 1 matches the key of token 0 as well as its
    own and hardly any other.  Token 1 ends the sequence; token 0 stands 19 places back (the last key a window of 20
    keeps) or 20 places back (the first it drops).  In a prompt, in portions that end at the edge, and decoded."""
    mixes, window = EDGES[case]
    cfg = _one_layer(*mixes)
    d = str(tmp_path / "edge")

    def edit(w):
        for i, (t, m) in enumerate(mixes):
            _plain_stream(w, f"l{i}.")
            if t == "attention":
                _edge_attention(w, f"l{i}.mix.")
            else:
                _edge_latent(w, f"l{i}.mix.", own="kv_from" not in m)
                if len(mixes) > 1 and i == 0:
                    w["l0.mix.o"] = torch.zeros_like(w["l0.mix.o"])     # the owner's own attention says nothing
        _twins(w)

    cfg, w = write_model(d, cfg=cfg, seed=11, edit=edit)
    rng = np.random.RandomState(0)
    for back in (window - 1, window):
        toks = rng.randint(2, 64, size=90).tolist()
        toks[-1 - back], toks[-1] = 0, 1
        ref = plain.forward(cfg, w, toks).numpy()
        other = list(toks)
        other[-1 - back] = 2
        moved = np.abs(ref[-1] - plain.forward(cfg, w, other).numpy()[-1]).max() / np.abs(ref[-1]).max()
        assert (moved > 0.1) == (back == window - 1), (back, moved)   # inside the window the key decides, outside it is gone
        for dtype in ("float32", "bfloat16"):
            reqs = {"a": toks}
            for steps in (helpers.trace_whole(reqs), helpers.trace_prefill_then_decode(reqs, tail=30),
                          helpers.trace_portions(reqs, sizes=(90 - back - 1, 2, back - 2, 1)),
                          helpers.trace_portions(reqs, sizes=(90 - back, back - 1, 1))):
                eng = engine_of(d, dtype, 4, 128)
                compare(helpers.replay(eng, steps), {"a": ref}, dtype, f"{case}, key {back} back")


@gpu
def test_pages_outlive_the_owners_window(models):
    """Rows read through windows of 24, 40 and 9 live in one cache group of the widest; it gives back what that one has
    passed."""
    d, cfg, w, reqs, ref, page = models["A", "float32"]
    eng = engine_of(d, "float32", page, 512)
    assert [g.window for g in eng.cache.groups] == [40, 17]
    eng.open_request("x")
    from ccinfer_b200.engine.engine import StepEntry
    eng.step([StepEntry("x", [1] * 100, [])])
    held = [p.used_pages for p in eng.cache.pools]
    assert held[0] == 13 - (100 - 40 + 1) // page and held[1] == 13 - (100 - 17 + 1) // page


@gpu
def test_a_sink_decides(tmp_path):
    """Sinks far above every score, in a latent layer with rows of its own and in one that reads them: most of each
    softmax's weight goes to the term that has no value."""
    cfg = plain.model(64, 32, 2, 1e-5, [(plain.latent(3, 8, 4, 8, 16, 12, 0.3, window=30), None),
                                        (plain.latent(2, 8, 4, 8, 16, 12, 0.3, window=8, kv_from=0), None)])
    d = str(tmp_path / "sink")
    sinks = {"l0.mix.sink": torch.tensor([4.0, 6.0, -1.0]), "l1.mix.sink": torch.tensor([5.0, 3.0])}
    cfg, w = write_model(d, cfg=cfg, seed=12, edit=lambda w: w.update(sinks))
    toks = np.random.RandomState(1).randint(0, 64, size=40).tolist()
    ref = plain.forward(cfg, w, toks).numpy()
    low = dict(w, **{k: torch.full_like(v, -30.0) for k, v in sinks.items()})
    assert np.abs(plain.forward(cfg, low, toks).numpy() - ref).max() > 0.1 * np.abs(ref).max()
    for dtype in ("float32", "bfloat16"):
        eng = engine_of(d, dtype, 4, 64)
        for steps in (helpers.trace_whole({"a": toks}), helpers.trace_prefill_then_decode({"a": toks}, tail=20)):
            compare(helpers.replay(eng, steps), {"a": ref}, dtype, "sink")


@gpu
def test_a_far_token_decides_through_the_state(tmp_path):
    """One delta layer that forgets nearly nothing.  q and k read the first half of the stream, v the second.  The keys of
    tokens 0 and 1 lie along the first coordinate and those of all others across it.  Token 0 stands at ONE far place among
    400 and token 1 at the end: what the state kept of the far token decides the last logits.  The far place is the first
    token, around a page border and the middle; the prompt is cut so that the state crosses steps."""
    cfg = _one_layer(plain.delta(2, 1, 16, 16, 2))
    d = str(tmp_path / "far")

    def edit(w):
        p = "l0.mix."
        _plain_stream(w, "l0.")
        w[p + "v"][:, :16] = 0
        w[p + "k"] = torch.eye(32)[:16] * 6.0
        w[p + "q"] = w[p + "k"].clone()
        for c in ("q.conv", "k.conv", "v.conv"):
            w[p + c] = torch.cat([0.1 * torch.ones_like(w[p + c][:, :1]), torch.ones_like(w[p + c][:, 1:])], 1)
        w[p + "A_log"] = torch.full((2,), -9.0)
        w[p + "dt_bias"] = torch.full((2,), -3.0)
        w[p + "a"] = torch.zeros_like(w[p + "a"])
        w[p + "b"] = torch.zeros_like(w[p + "b"])
        w["embed"][:2, :16] = torch.tensor([4.0] + 15 * [-1.0])
        w["embed"][2:, :16] = 2.0 * w["embed"][2:, :16].abs()
        w["embed"][2:, 0] = -1.0
        w[p + "o"] *= 3.0

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
                compare(helpers.replay(eng, steps), {"a": ref}, dtype, f"far token at {far_at}")


@gpu
def test_the_first_tap_decides_across_portions(tmp_path):
    """A convolution of four taps whose oldest weighs most: the input three tokens back decides, whether it came with the
    same portion, an earlier one, or a decoded token; the ring's place is used again every four positions."""
    cfg = _one_layer(plain.delta(2, 2, 8, 8, 4))
    d = str(tmp_path / "taps")

    def edit(w):
        _plain_stream(w, "l0.")
        for c in ("q.conv", "k.conv", "v.conv"):
            w["l0.mix." + c] = torch.cat([torch.full_like(w["l0.mix." + c][:, :1], 3.0), 0.2 * w["l0.mix." + c][:, 1:]], 1)

    cfg, w = write_model(d, cfg=cfg, seed=3, edit=edit)
    reqs = requests_of(cfg, [1, 2, 3, 4, 5, 8, 9, 30], 4)
    ref = {rid: plain.forward(cfg, w, t).numpy() for rid, t in reqs.items()}
    for dtype in ("float32", "bfloat16"):
        bounds = bounds_of(cfg, w, reqs, ref, dtype)
        for sizes in ((1,), (2,), (3,), (4, 1), (1, 5, 2), (2, 1, 1, 7)):
            eng = engine_of(d, dtype, 4, 64)
            compare(helpers.replay(eng, helpers.trace_portions(reqs, sizes=sizes)), ref, dtype, f"taps, portions {sizes}", bounds)


@gpu
def test_long_decoding(models):
    """260 tokens one by one: the windows pass over decoded tokens many times, their pages are given back."""
    rng = np.random.RandomState(9)
    for dtype in ("float32", "bfloat16"):
        d, cfg, w, reqs, ref, page = models["A", dtype]
        toks = rng.randint(0, cfg["vocab"], size=260).tolist()
        want = plain.forward(cfg, w, toks).numpy()
        eng = engine_of(d, dtype, page, 320, use_graphs=(dtype == "bfloat16"))
        rows = helpers.replay(eng, helpers.trace_prefill_then_decode({"a": toks}, tail=10 ** 6))
        worst = compare(rows, {"a": want}, dtype, f"long decoding {dtype}", bounds_of(cfg, w, {"a": toks}, {"a": want}, dtype))
        print(f"[worst] long decoding, {dtype}: {worst:.3e}")
        assert all(p.high_water <= 40 // page + 2 for p in eng.cache.pools)


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(models, dtype):
    """Prompts of unequal length in portions of 7 through ``LLM.generate`` and its scheduler, which launches a step before
    the tokens of the step before it have been read: the tables' experts are found by tokens still on the device."""
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
                assert row[t] >= row.max() - 0.05 * row.abs().max()
                toks.append(t)
    assert all(pool.used_pages == 0 for pool in llm.engine.cache.pools)


@gpu
def test_a_preempted_request_starts_its_state_again(models):
    """So few pages that a request is preempted and computed again (its slot is closed and opened: the recurrent state
    starts again, the pages are taken anew): the greedy tokens are those of a calm run."""
    from ccinfer_b200 import LLM, SamplingParams
    d, cfg, w, reqs, ref, page = models["B", "float32"]
    rng = np.random.RandomState(6)
    prompts = [rng.randint(0, cfg["vocab"], size=n).tolist() for n in (20, 26, 17)]
    llm = LLM(d, dtype="float32", page_size=page, kv_tokens=16 * page, prefill_chunk_size=16, max_requests=4,
              max_tokens_per_step=64)
    got = llm.generate(prompts, [SamplingParams(max_tokens=n) for n in (24, 20, 28)])
    assert llm.scheduler.preemptions > 0
    assert got == [plain.greedy(cfg, w, p, n) for p, n in zip(prompts, (24, 20, 28))]
    llm.engine.cache.check_consistency()


@gpu
def test_the_programs_as_a_user_calls_them(models, tmp_path):
    """bin/ccinfer: greedy tokens of a model folder; a random model written from a configuration generates the same tokens
    as the same configuration drawn on the device; bin/trace_run: a mixed trace over four request slots, its files
    against the plain logits."""
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    d, cfg, w, reqs, ref, page = models["A", "float32"]
    exe = [sys.executable, os.path.join(root, "bin", "ccinfer")]
    prompt = list(reqs.values())[12]
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
    assert len(a.stdout.strip().splitlines()) == len(b.stdout.strip().splitlines()) == 2

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
