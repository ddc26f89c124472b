"""Latent attention: keys and values of all heads made from one low-rank vector per token.

With H heads of ``dim`` unrotated and ``rot_dim`` rotated query/key coordinates, value size ``vdim`` and latent
size ``rank``:

    q = Wq x                      [H, dim | rot_dim]
    [c' | kr'] = Wdkv x           c = c' / rms(c') * w_c  (rank),  kr = rot(kr')  (rot_dim, one for all heads)
    k_h = [Wuk_h c | kr],  v_h = Wuv_h c
    s_ij = (q_h,i . k_h,j) * scale  for  0 <= i - j < window;   p = exp(s) / (sum_j exp(s_ij) + exp(sink_h))
    o_h = sigmoid(Wg x)_h * sum_j p_ij v_h,j;   out = Wo [o_1 .. o_H]

The rotation turns the pairs (i, i + rot.dims / 2) of the first ``rot.dims`` rotated coordinates of q and of kr
by position * base^(-2i / rot.dims); with ``interleaved`` the pairs are (2i, 2i + 1) instead, which the kernels see as
the same thing after the rows of Wq's rotated parts and of Wdkv's are permuted alike when they are bound (a score
does not change when q and k are permuted alike).  ``window`` None: every earlier token is seen.  Without a gate
tensor the heads' results are taken as they are.  ``own_kv`` False: the layer has no Wdkv and reads the rows that
another layer of the same latent size, rotated size and rotation left in its cache.  ``q_rank`` N: the queries go
through a latent vector of their own, q = Wuq (c_q / rms(c_q) * w_q) with c_q = Wdq x (N coordinates).  ``ramp_scaling``:
slow pairs turn slower and cosine and sine carry a factor, as ``position.RotaryHalf`` has it.

What a token leaves in the cache is the row [c | kr] alone.  Attention runs over those rows: the unrotated part
of a query is carried into the latent space first, (Wuk_h^T q_h) . c = q_h . (Wuk_h c), and the weighted sum of c
comes back out through Wuv_h afterwards (two products per head, batched over the heads).  q (or c_q), the latent row
and the gate are ONE merged product of x.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..errors import Unsupported
from .base import CachedTensor, CacheNeed, Mixer, TensorSpec
from .position import RotaryHalf


def _pad8(n: int) -> int:
    return -(-n // 8) * 8


class LatentAttention(Mixer):
    kernel_groups = ("latent",)
    def __init__(self, hidden: int, heads: int, dim: int, rot_dim: int, value_dim: int, rank: int, window: int,
                 scale: float, rot_base: float, rot_dims: int, norm_eps: float, names: dict,
                 interleaved: bool = False, own_kv: bool = True, q_rank: int = None, ramp_scaling: dict = None):
        """``names``: tensor names under the keys q (with ``q_rank`` dq, dq_norm, uq instead), dkv, dkv_norm, uk, uv, sink,
        o and optionally g (the gate)."""
        if window is not None and window <= 0:
            raise Unsupported("a window of keys is > 0 (None: every earlier token)")
        if rot_dims % 2 or not (0 <= rot_dims <= rot_dim):
            raise Unsupported(f"rotation of {rot_dims} of {rot_dim} coordinates: even, at most rot_dim")
        if rank > 1024:
            raise Unsupported(f"latent size {rank}: the attention kernel holds up to 1024 coordinates per warp")
        self.hidden, self.H, self.d, self.r, self.dv, self.R = (int(hidden), int(heads), int(dim), int(rot_dim),
                                                                int(value_dim), int(rank))
        self.window = int(window) if window is not None else None
        self.kernel_window = self.window if self.window is not None else 2 ** 31 - 1   # (what the kernels are told)
        self.scale, self.eps = float(scale), float(norm_eps)
        self.rot_base, self.rot_dims = float(rot_base), int(rot_dims)
        self.interleaved, self.own_kv = bool(interleaved), bool(own_kv)
        self.names = dict(names)
        self.has_gate = "g" in self.names
        self.q_rank = int(q_rank) if q_rank is not None else None
        self.ramp_scaling = dict(ramp_scaling) if ramp_scaling is not None else None
        self.q_width = self.H * (self.d + self.r)
        # columns of the merged product: q or c_q | [c' | kr'] | gate logits, each start a multiple of 8
        self.oq = 0
        self.oc = _pad8(self.q_width if self.q_rank is None else self.q_rank)
        self.og = self.oc + (_pad8(self.R + self.r) if self.own_kv else 0)
        self.in_width = self.og + (_pad8(self.H) if self.has_gate else 0)
        self.rt = None

    def tensor_specs(self):
        n, D, H = self.names, self.hidden, self.H
        if self.q_rank is None:
            specs = [TensorSpec(n["q"], (self.q_width, D))]
        else:
            specs = [TensorSpec(n["dq"], (self.q_rank, D)),
                     TensorSpec(n["dq_norm"], (self.q_rank,), role="vector", init="one_plus_normal"),
                     TensorSpec(n["uq"], (self.q_width, self.q_rank))]
        specs += [TensorSpec(n["uk"], (H * self.d, self.R)), TensorSpec(n["uv"], (H * self.dv, self.R)),
                  TensorSpec(n["sink"], (H,), role="vector"), TensorSpec(n["o"], (D, H * self.dv))]
        if self.own_kv:
            specs += [TensorSpec(n["dkv"], (self.R + self.r, D)),
                      TensorSpec(n["dkv_norm"], (self.R,), role="vector", init="one_plus_normal")]
        if self.has_gate:
            specs.append(TensorSpec(n["g"], (H, D)))
        return specs

    def cache_need(self):
        return CacheNeed((CachedTensor("latent", (self.R + self.r,), token_axis=0),), self.window)

    def bind(self, rt, fetch):
        self.rt = rt
        n, H = self.names, self.H
        w = torch.zeros((self.in_width, self.hidden), dtype=rt.dtype, device=rt.device)
        # the rotated coordinates in the kernels' order: pair i at places (i, i + rot_dims / 2)
        perm = None
        if self.interleaved and self.rot_dims:
            half = self.rot_dims // 2
            perm = torch.tensor([2 * i for i in range(half)] + [2 * i + 1 for i in range(half)]
                                + list(range(self.rot_dims, self.r)), device=rt.device)
        wq = fetch(n["q"] if self.q_rank is None else n["uq"])
        if perm is not None:
            wq = wq.view(H, self.d + self.r, -1).clone()
            wq[:, self.d:] = wq[:, self.d:][:, perm]
            wq = wq.view(H * (self.d + self.r), -1)
        if self.q_rank is None:
            w[self.oq:self.oq + wq.shape[0]] = wq
        else:
            t = fetch(n["dq"])
            w[self.oq:self.oq + t.shape[0]] = t
            self.cq_norm_w = fetch(n["dq_norm"]).float().contiguous()
            # (rows of c_q are padded with zeros to a multiple of 8, and so are this matrix's columns)
            self.w_uq = torch.zeros((_pad8(self.q_width), _pad8(self.q_rank)), dtype=rt.dtype, device=rt.device)
            self.w_uq[:wq.shape[0], :self.q_rank] = wq
        if self.own_kv:
            wc = fetch(n["dkv"])
            if perm is not None:
                wc = wc.clone()
                wc[self.R:] = wc[self.R:][perm]
            w[self.oc:self.oc + wc.shape[0]] = wc
        if self.has_gate:
            t = fetch(n["g"])
            w[self.og:self.og + t.shape[0]] = t
        self.w_in = w
        self.norm_w = (fetch(n["dkv_norm"]).float().contiguous() if self.own_kv
                       else torch.ones(self.R, dtype=torch.float32, device=rt.device))
        self.sink = fetch(n["sink"]).float().contiguous()
        # per head: [rank, dim] so that (q_h Wuk_h) is a product with the weights' usual layout [out, in]
        self.w_uk_t = fetch(n["uk"]).view(H, self.d, self.R).transpose(1, 2).contiguous()
        self.w_uv = fetch(n["uv"]).view(H, self.dv, self.R).contiguous()
        self.w_o = fetch(n["o"])
        self.inv_freq, self.amp = None, 1.0
        if self.rot_dims:
            rot = RotaryHalf(self.rot_dims, self.rot_base, ramp_scaling=self.ramp_scaling,
                             linear_scaling=1.0 if self.ramp_scaling is None else None)   # (1: evaluated in float64)
            rot.bind(rt, fetch)
            self.inv_freq = rot.rotary_table()
            amp = rot.amplitude()
            self.amp = 1.0 if amp is None else float(amp[0])

    def forward(self, x, step, cache, state):
        rt = self.rt
        x = rt.rows(x)
        T = x.shape[0]
        H, d, r, R, dv = self.H, self.d, self.r, self.R, self.dv
        g = cache.group
        proj = rt.scratch.get("latent_proj", (rt.max_tokens, self.in_width), rt.dtype)[:T]
        rt.linear(proj, x, self.w_in)
        qa = rt.scratch.get("latent_q", (rt.max_tokens, H, R + r), torch.float32)[:T]
        rows = cache.tensors["latent"]
        prepare = (self.oc, self.norm_w, self.inv_freq, self.rot_dims, step.positions, g.slot_map if cache.own else None,
                   rows, H, d, r, R, self.eps)
        if self.q_rank is None:
            q = proj[:, self.oq:self.oq + self.q_width]
            kernels.latent_prepare(proj, *prepare, q=q, qa=qa, amp=self.amp, status=rt.status)
        else:
            cq = rt.scratch.get("latent_cq", (rt.max_tokens, self.w_uq.shape[1]), rt.dtype)[:T]
            kernels.latent_prepare(proj, *prepare, amp=self.amp, low=(self.oq, self.q_rank, self.cq_norm_w, cq),
                                   status=rt.status)
            q = rt.scratch.get("latent_uq", (rt.max_tokens, self.w_uq.shape[0]), rt.dtype)[:T]
            rt.linear(q, cq, self.w_uq)
            kernels.latent_prepare(q, *prepare[:5], None, None, *prepare[7:], q=q, qa=qa, amp=self.amp, status=rt.status)
            q = q[:, :self.q_width]
        if d > 0:
            qu = q.view(T, H, d + r)[:, :, :d]
            rt.linear_batched(qa[:, :, :R].permute(1, 0, 2), qu.permute(1, 0, 2), self.w_uk_t)
        else:
            qa[:, :, :R].zero_()
        ol = rt.scratch.get("latent_o", (rt.max_tokens, H, R), rt.dtype)[:T]
        gate = proj[:, self.og:self.og + H] if self.has_gate else None
        args = (qa, rows, self.sink, gate, ol, step.cu_q, step.pos0, step.entry_of_token, g.block_table)
        n1, many = step.n_single, step.n_entries - step.n_single
        if kernels.latent_attention_mma_fits(rt.dtype, R, r):
            # tensor cores: the heads are the rows of the products.  The step's single tokens come first; their
            # key ranges are cut into pieces so that a few rows still fill the machine
            if n1 > 0:
                splits = kernels.latent_attention_splits(n1, H, self.kernel_window)
                acc = ml = None
                if splits > 1:
                    most = kernels.latent_attention_splits(1, H, self.kernel_window)   # (rows x pieces is bounded by the target)
                    cap = max(rt.max_entries * H * most, kernels.split_target_blocks() * kernels.LATENT_MMA_ROWS * 2)
                    acc = rt.scratch.get("latent_part_acc", (cap * R,), torch.float32)
                    ml = rt.scratch.get("latent_part_ml", (cap * 2,), torch.float32)
                kernels.latent_attention_mma(*args, 0, n1, 1, g.page_size, self.kernel_window, self.scale, splits, acc, ml,
                                             status=rt.status)
            if many > 0:
                kernels.latent_attention_mma(*args, n1, many, step.max_q_len, g.page_size, self.kernel_window, self.scale,
                                             status=rt.status)
        else:   # the plain kernel: float, and sizes that are multiples of nothing
            if n1 > 0:
                kernels.latent_attention(*args, 0, n1, 1, g.page_size, self.kernel_window, self.scale, status=rt.status)
            if many > 0:
                kernels.latent_attention(*args, n1, many, step.max_q_len, g.page_size, self.kernel_window, self.scale,
                                         status=rt.status)
        o = rt.scratch.get("latent_v", (rt.max_tokens, H, dv), rt.dtype)[:T]
        rt.linear_batched(o.permute(1, 0, 2), ol.permute(1, 0, 2), self.w_uv)
        out = rt.scratch.get(self.out_key, (rt.max_tokens, self.hidden), rt.dtype)[:T]
        return rt.linear(out, o.view(T, H * dv), self.w_o)
