"""Differential attention (Ye et al. 2024, "Differential Transformer") with grouped keys over the paged cache: two softmax
maps per head over the same values, the second subtracted from the first.

   q = W_q h  (heads x 2 x key_dim),  k = W_k h  (kv_heads x 2 x key_dim),  v = W_v h  (kv_heads x value_dim)
   every query and key of every map: divided by its root mean square, times a weight [key_dim] (``qk_norm``), then the
       first ``position.rotary_dim`` numbers are rotated (position part: frequencies); the rest pass
   s_m[i, j] = scale * q_(h,m)[i] . k_(g,m)[j]     for j <= i, and j // chunk = i // chunk where there is a chunk
   a_m = softmax_j(s_m) v_g;   lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff
   o = a_1 - lambda a_2,   o <- o / sqrt(mean(o^2) + eps) * (1 - diff)      over the head's value_dim numbers
   y = W_o concat_h(o_h)
Query head h reads kv head h // (num_heads / num_kv_heads).  The cache keeps pages of the normed and rotated k
(2 kv_heads vectors) and of v.  With ``own_keys`` off the mixer has no keys and values of its own and reads those that
another layer wrote to its cache slot in the same step; ``held`` says how far back that slot's readers look:
(window, whether it is a chunk), or None for everything.  Angles, scores, weights, sums and the last norm are 32-bit in both
precisions; lambda is formed once after loading, in 64-bit.
"""
from __future__ import annotations

import math
from typing import Dict, Optional, Tuple

import torch

from .. import native
from . import registry
from .base import ProjectedMixer
from .conv_attention import attend, rotation_options, window_plan
from .registry import register
from .spec import CacheEntry, CacheNeed, ParamSpec, PartSpec


@register("mixer", "differential_attention")
class DifferentialAttention(ProjectedMixer):
    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, key_dim: int, value_dim: int, scale: float,
                 diff: float, norm_eps: float, position: Optional[PartSpec] = None, chunk: Optional[int] = None,
                 qk_norm: bool = True, own_keys: bool = True, held: Optional[Tuple[int, bool]] = None):
        if num_heads % num_kv_heads:
            raise ValueError("differential_attention: num_heads must be a multiple of num_kv_heads")
        if value_dim > 512 or key_dim > 4096:
            raise ValueError(f"differential_attention: sizes {key_dim} / {value_dim} are beyond what the kernels take (4096 / 512)")
        self.hidden_size, self.nh, self.nkv, self.dk, self.dv = hidden_size, num_heads, num_kv_heads, key_dim, value_dim
        self.scale, self.diff, self.norm_eps = float(scale), float(diff), float(norm_eps)
        # (a chunk beyond any context is one that never ends; the kernels take 32-bit sizes)
        self.chunk = min(int(chunk), 1 << 30) if chunk else None
        self.qk_norm, self.own_keys = bool(qk_norm), bool(own_keys)
        self.held = (min(int(held[0]), 1 << 30), bool(held[1])) if held else None
        self.position = registry.build("position", position) if position is not None else None
        if self.position is not None and not hasattr(self.position, "frequencies"):
            raise ValueError("differential_attention rotates by frequencies (a position part with ``frequencies``)")
        if self.position is not None and self.position.rotary_dim > key_dim:
            raise ValueError("differential_attention: rotary_dim exceeds key_dim")
        self.inner_cols = num_heads * value_dim

    def segments(self):
        q, k, v = 2 * self.nh * self.dk, 2 * self.nkv * self.dk, self.nkv * self.dv
        return {"qkv": (q, k, v) if self.own_keys else (q,)}

    def inner_params(self) -> Dict[str, ParamSpec]:
        p = {"lambdas": ParamSpec((4, self.dk), role="vector", init="normal", rows=(1, 1, 1, 1), members_lack_axis=True)}
        if self.qk_norm:
            p["q_norm"] = ParamSpec((self.dk,), role="vector", init="norm")
            if self.own_keys:
                p["k_norm"] = ParamSpec((self.dk,), role="vector", init="norm")
        return p

    def cache_need(self) -> CacheNeed:
        window, chunked = self.held if self.held else (None, False)
        return CacheNeed("pages", window=window, chunked=chunked,
                         entries=(CacheEntry("k", (2 * self.nkv, self.dk)), CacheEntry("v", (self.nkv, self.dv))))

    def after_load(self) -> None:
        lq1, lk1, lq2, lk2 = self.w_lambdas.double().cpu()
        self._lambda = math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + self.diff
        self._norms = None
        if self.qk_norm:
            wq, wk = self.w_q_norm, self.w_k_norm if self.own_keys else None
            if wk is not None and wk.dtype != wq.dtype:       # (a checkpoint may hold one of them in 32-bit)
                wq, wk = wq.float(), wk.float()
            self._norms = (wq, wk, self.norm_eps)

    def launch_plan(self, step):
        return window_plan(step, self.nh, self.nkv, self.dk, self.dv, self.chunk, 0, self.rt.dtype, maps=2)

    def inner(self, x, proj, step, cache, writes_cache, y, y_scale):
        T = y.shape[0]
        ws, dt = self.rt.workspace, self.rt.dtype
        nh, nkv, dk, dv = self.nh, self.nkv, self.dk, self.dv
        pos = self.position
        freq = pos.frequencies(self.rt) if pos is not None and pos.rotary_dim else None
        q = ws.get("da.q", (T, 2 * nh * dk), dt)
        writes = writes_cache and self.own_keys
        native.conv_rope_write(q, proj["qkv"], 2 * nh, 2 * nkv if self.own_keys else 0, dk, dv, None, None, freq,
                               pos.rotary_dim if freq is not None else 0, step.positions, step.seq_of_token, step.cu_q,
                               step.state_slots, step.block_tables[cache.group], cache.page_size,
                               cache.k_pages if writes else None, cache.v_pages if writes else None, step.status,
                               value_heads=nkv if self.own_keys else 0, head_norms=self._norms, **rotation_options(pos))
        attend(self.launch_plan(step), ws, y, q, cache, step, nh, nkv, dk, dv, self.scale, 0.0, self.chunk, 0,
               out_scale=y_scale * (1.0 - self.diff), chunked=self.chunk is not None, maps=(self._lambda, self.norm_eps))
