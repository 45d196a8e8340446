"""Differential attention over the cache, as a mixer: every head has ``maps`` = 2 queries and two
keys over the same values. Each map is a causal softmax attention of its own, with an optional
window; with their outputs a_1 and a_2 the head gives

    o = a_1 - lambda a_2,   o / sqrt(mean(o^2) + eps) * (1 - diff),
    lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff

(lambda is one number of the layer, formed once at load). q, k and v have biases; q and k are
normed per map with one weight for all heads and maps, then rotated. One product gives the rows
[q | k | v]; one kernel adds the biases, norms, rotates and stores keys and values; one
attention kernel does both maps, their difference and the norm over the head.

A row of the cache holds a key head's two maps one after the other (``head_dim`` = 2 dim), so
that a page of keys is one tile for both.
"""
from __future__ import annotations

import math
from typing import Dict, List

import torch

from .. import kernels as K
from ..errors import ConfigError, KernelError
from .base import MIXERS, CacheNeed, Part, TensorNeed
from .linear import Linear, Pending


class DifferentialAttention(Part):
    capturable = True
    can_store = True      # forward(..., store=True) writes its output into x instead of adding

    def __init__(self, spec, prefix: str = "", positions=None):
        super().__init__(spec, prefix)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.nh, self.nkv = int(p["heads"]), int(p["kv_heads"])
        if self.nkv <= 0 or self.nh % self.nkv:
            raise ConfigError(f"{self.nh} heads on {self.nkv} KV heads")
        self.dim, self.vd = int(p["dim"]), int(p["vdim"])
        self.window = int(p.get("window", 0))
        self.scale, self.diff, self.eps = float(p["scale"]), float(p["diff"]), float(p["eps"])
        self.position = (positions or {}).get(p.get("position", ""))
        if p.get("position") and self.position is None:
            raise ConfigError(f"the mixer names the position encoding \"{p['position']}\", "
                              "which the model does not define")
        self.names = {k: prefix + v for k, v in p["names"].items()}
        self.qw, self.kw, self.vw = 2 * self.nh * self.dim, 2 * self.nkv * self.dim, self.nkv * self.vd
        self.ow = self.nh * self.vd

    def libraries(self, rt) -> List[str]:
        return ["rope", "attention_diff"] + (["attention_diff_tc"] if rt.fast_kernels else [])

    def tensors(self) -> List[TensorNeed]:
        n, d = self.names, self.dim
        return [TensorNeed(n["q"], (self.qw, self.hidden)),
                TensorNeed(n["q_bias"], (self.qw,), "bias"),
                TensorNeed(n["k"], (self.kw, self.hidden)),
                TensorNeed(n["k_bias"], (self.kw,), "bias"),
                TensorNeed(n["v"], (self.vw, self.hidden)),
                TensorNeed(n["v_bias"], (self.vw,), "bias"),
                TensorNeed(n["q_norm"], (d,), "vector"), TensorNeed(n["k_norm"], (d,), "vector"),
                TensorNeed(n["lq1"], (d,), "bias"), TensorNeed(n["lk1"], (d,), "bias"),
                TensorNeed(n["lq2"], (d,), "bias"), TensorNeed(n["lk2"], (d,), "bias"),
                TensorNeed(n["o"], (self.hidden, self.ow))]

    def cache_need(self) -> CacheNeed:
        return CacheNeed(self.nkv, 2 * self.dim, self.window, 2,
                         0 if self.vd == 2 * self.dim else self.vd)

    def bind(self, weights: Dict[str, torch.Tensor], rt) -> None:
        self.rt = rt
        if self.dim > K.DIFF_MAX_DIM or self.vd > K.DIFF_MAX_VDIM:
            raise KernelError(f"maps of {self.dim} values and value rows of {self.vd} are not "
                              "supported by the differential attention kernels (at most "
                              f"{K.DIFF_MAX_DIM} and {K.DIFF_MAX_VDIM})")
        n = self.names
        w = [weights[n[k]] for k in ("q", "k", "v")]
        if len({t.dtype for t in w}) > 1:
            w = [t.float() for t in w]
        self.qkv = Linear(torch.cat(w, dim=0), rt)
        if getattr(rt, "consume_weights", False):
            del w
            for key in ("q", "k", "v"):
                weights.pop(n[key], None)
        self.bias = torch.cat([weights[n[k]].to(torch.float32)
                               for k in ("q_bias", "k_bias", "v_bias")]).contiguous()
        self.q_norm = weights[n["q_norm"]].to(torch.float32).contiguous()
        self.k_norm = weights[n["k_norm"]].to(torch.float32).contiguous()
        dot = lambda a, b: float((weights[n[a]].double() * weights[n[b]].double()).sum())
        self.lam = math.exp(dot("lq1", "lk1")) - math.exp(dot("lq2", "lk2")) + self.diff
        self.o = Linear(weights[n["o"]], rt)

    def forward(self, h, x, step, line, state, writes_cache: bool, store: bool = False):
        """Adds the mixer's output into x (``store``: writes it there), or returns it as
        ``Pending`` split sums, with x left as it is."""
        if not writes_cache:
            raise ConfigError("differential attention writes the cache line that it reads")
        T = h.shape[0]
        inv_freq, rot_dim = (self.position.frequencies() if self.position is not None
                             else (None, 0))
        amplitude = self.position.amplitude if self.position is not None else 1.0
        # split sums are added up by the kernel that norms and rotates
        rows = self.qkv(h, defer=True)
        rows = rows.partial if isinstance(rows, Pending) else rows
        q = torch.empty((T, self.qw), dtype=self.rt.dtype, device=h.device)
        K.maps_norm_rope_store(rows, self.bias, self.q_norm, self.k_norm, self.eps, inv_freq,
                               rot_dim, amplitude, step, line, self.nh, self.nkv, 2, self.dim,
                               self.vd, q)
        attn = torch.empty((T, self.ow), dtype=self.rt.dtype, device=h.device)
        self.rt.differential_attention(q, attn, step, line, self.nh, self.nkv, self.dim, self.vd,
                                       self.window, self.scale, self.lam, 1.0 - self.diff,
                                       self.eps)
        out = self.o(attn, out=x, defer="any") if store else self.o(attn, add_into=x, defer=True)
        return out if isinstance(out, Pending) else None


MIXERS.register("differential_attention", DifferentialAttention)
