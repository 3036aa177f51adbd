"""Mixer ``latent_attention``: causal attention whose keys and values come from one low-rank latent per token.

Per token the layer computes, from its input h:

* a query latent, RMS-normed, expanded to H heads of ``dim`` plain + ``rot_dim`` rotated entries — or, with ``q_rank`` 0,
  the heads straight from h;
* a key/value latent c of rank ``kv_rank``, RMS-normed, and ONE rotated key part r of ``rot_dim`` entries that all heads
  share (not normed);
* head h's key is [Uk_h c | r], its value Uv_h c; score = (q_plain . Uk_h c + q_rot . r) * scale; softmax; W_o.

Only [c | r] is cached: one row of kv_rank + rot_dim entries per token (a key-only cache group with one head).  The
expansions are folded into the query and the output, (Uk_hᵀ q_plain) . c and Uv_h (Σ p c), so that attention runs over
the cached rows directly, the same way for a prompt and for a single token.  Norms, scores, softmax and the rotation's
angles are fp32; the rotation turns the first ``rot_dims`` entries of the rotated part, pair i by the angle
pos * base^(-2i/dims): neighbouring entries (2i, 2i+1) (``pairing`` 1) or entries (i, i + dims/2) (``pairing`` 0) — or as a
position part says (its frequencies, pairing and amplitude).  With a
``window`` a query sees the last ``window`` positions only, and the cache gives pages before it back.  A mixer with
``shares_kv`` has no down-projection for keys and values: its call reads the rows another call's cache holds (``cache_of`` in
the schedule) with its own queries and expansions.
"""
from __future__ import annotations

import numpy as np
import torch

from ..cache.storage import KVRequest
from ..ops import kernels
from .registry import TensorDecl, nested_build, nested_declare, part


@part("mixer", "latent_attention")
class LatentAttention:
    """params: ``width``, ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``kv_rank``, ``q_rank``, ``scale``, ``rot_base``,
    ``rot_dims`` (how many of the rot_dim entries are rotated), ``eps`` (of the RMS norms), optional ``pairing`` (default 1)
    and ``window`` (0: every earlier position); ``position`` (a PartSpec of the position family, instead of ``rot_base``,
    ``rot_dims`` and ``pairing``); ``shares_kv`` (default False; the tensors ``dkv`` and ``dkv.norm`` are absent then).
    tensors: ``dq`` [q_rank, width], ``dq.norm`` [q_rank], ``uq`` [heads*(dim+rot_dim), q_rank] (with q_rank 0 instead of
    these three ``q`` [heads*(dim+rot_dim), width]), ``dkv`` [kv_rank+rot_dim,
    width], ``dkv.norm`` [kv_rank], ``uk`` [heads*dim, kv_rank], ``uv`` [heads*vdim, kv_rank], ``o`` [width, heads*vdim]."""
    stores_output = True
    scales_output = True
    defers_norm = True       # the input may be a deferred norm, and the output projection can fill the next one

    @classmethod
    def declare(cls, spec):
        p = spec.params
        W, H, D, R, Dv, C, Q = p["width"], p["heads"], p["dim"], p["rot_dim"], p["vdim"], p["kv_rank"], p["q_rank"]
        queries = ({"dq": TensorDecl((Q, W)), "dq.norm": TensorDecl((Q,), "norm_scale"), "uq": TensorDecl((H * (D + R), Q))}
                   if Q else {"q": TensorDecl((H * (D + R), W))})
        rows = {} if p.get("shares_kv", False) else {"dkv": TensorDecl((C + R, W)), "dkv.norm": TensorDecl((C,), "norm_scale")}
        turned = nested_declare("position", p["position"]) if p.get("position") is not None else {}
        return {**queries, **rows, "uk": TensorDecl((H * D, C)), "uv": TensorDecl((H * Dv, C)), "o": TensorDecl((W, H * Dv)), **turned}

    def __init__(self, spec, tensors, rt, **_):
        p = spec.params
        self.rt = rt
        self.width, self.H, self.D, self.R = int(p["width"]), int(p["heads"]), int(p["dim"]), int(p["rot_dim"])
        self.Dv, self.C, self.Q = int(p["vdim"]), int(p["kv_rank"]), int(p["q_rank"])
        self.scale, self.eps = float(p["scale"]), float(p["eps"])
        self.window, self.amplitude = int(p.get("window", 0)), 1.0
        if p.get("position") is not None:
            position = nested_build("position", p["position"], tensors, rt)
            self.rot_dims, self.pairing = int(position.rotary_dim), int(position.pairing)
            self.inv_freq, self.amplitude = position.inv_freq, float(position.amplitude)
        else:
            self.rot_dims, self.pairing = int(p.get("rot_dims", self.R)), int(p.get("pairing", 1))
            i = np.arange(self.rot_dims // 2, dtype=np.float64)
            inv = np.power(np.float64(p["rot_base"]), -2.0 * i / max(self.rot_dims, 1)).astype(np.float32)
            self.inv_freq = torch.from_numpy(inv).to(rt.device) if inv.size else None
        if self.rot_dims % 2 or self.rot_dims > self.R:
            raise ValueError("latent_attention: rot_dims must be even and at most rot_dim")
        if self.inv_freq is None:
            self.inv_freq = torch.zeros(1, dtype=torch.float32, device=rt.device)
        self.shares_kv = bool(p.get("shares_kv", False))
        if self.shares_kv and not self.Q:
            raise ValueError("latent_attention: a mixer on another layer's rows makes its queries through a latent")
        # one product for what reads h: rows [query latent, or the queries themselves | kv latent | shared key part]
        names = ["dq" if self.Q else "q"] + ([] if self.shares_kv else ["dkv"])
        self.w_down = rt.to_compute(torch.cat([tensors[n] for n in names], dim=0))
        self.w_cnorm = None if self.shares_kv else rt.to_f32(tensors["dkv.norm"])
        self.w_qnorm = rt.to_f32(tensors["dq.norm"]) if self.Q else None
        self.w_uq = rt.to_compute(tensors["uq"]) if self.Q else None
        # per head: Uk_hᵀ [C, D] (folded into the query) and Uv_h [Dv, C] (applied to the context)
        self.w_uk_t = rt.to_compute(tensors["uk"].reshape(self.H, self.D, self.C).transpose(1, 2).contiguous())
        self.w_uv = rt.to_compute(tensors["uv"].reshape(self.H, self.Dv, self.C).contiguous())
        self.w_o = rt.to_compute(tensors["o"])

    def cache_request(self):
        return KVRequest(1, self.C + self.R, self.window, values=False)

    def weight_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.w_down, self.w_uq, self.w_uk_t, self.w_uv, self.w_o) if t is not None)

    @property
    def takes_padding_rows(self) -> bool:
        return True          # every kernel skips token rows of no sequence

    def forward(self, h, x, ctx, binding, store: bool = False, then_norm=None, out_scale=None) -> bool:
        T = h.shape[0]
        if binding.writes == self.shares_kv:
            raise ValueError("latent_attention: a layer without a down-projection for keys and values must read another "
                             "call's cache, and only such a layer may")
        rt, H, D, R, C, Q, Dv = self.rt, self.H, self.D, self.R, self.C, self.Q, self.Dv
        g = binding.group
        pages = ctx.pages_of(g)
        cache = g.k[binding.index]
        down = rt.scratch("latent_down", (T, self.w_down.shape[0]), torch.float32)
        kernels.linear(h, self.w_down, down, None, kernels.OUT_STORE_F32)
        qa = rt.scratch("latent_qa", (T, H * (C + R)))
        if Q:
            cq = rt.scratch("latent_cq", (T, Q))
            kernels.latent_prepare(down, Q, C, R, self.w_qnorm, self.w_cnorm, self.eps, self.inv_freq, self.rot_dims, ctx, pages,
                                   g.page_size, cache, cq, write_kv=binding.writes, pairing=self.pairing, amplitude=self.amplitude)
            q = rt.scratch("latent_q", (T, H * (D + R)))
            kernels.linear(cq, self.w_uq, q)
            kernels.linear_batched(q, D + R, self.w_uk_t, qa, C + R, D)
            kernels.latent_q_rotate(q, D, qa, C, R, H, self.inv_freq, self.rot_dims, ctx, self.pairing, self.amplitude)
        else:
            qn = rt.scratch("latent_q", (T, H * D))
            kernels.latent_prepare_direct(down, H, D, C, R, self.w_cnorm, self.eps, self.inv_freq, self.rot_dims, self.pairing, ctx,
                                          pages, g.page_size, cache, qn, qa, write_kv=binding.writes, amplitude=self.amplitude)
            kernels.linear_batched(qn, D, self.w_uk_t, qa, C + R, D)
        lat = rt.scratch("latent_ctx", (T, H * C))
        kernels.attention_latent(qa, lat, cache, ctx, pages, g.page_size, H, C, R, self.scale, rt=rt, window=self.window)
        heads = rt.scratch("attn_out", (T, H * Dv))
        kernels.linear_batched(lat, C, self.w_uv, heads, Dv, C)
        return kernels.linear(heads, self.w_o, x, None, kernels.OUT_STORE_F32 if store else kernels.OUT_ADD_F32,
                              None if store else then_norm, out_scale)
