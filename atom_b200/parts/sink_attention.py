"""Grouped-query attention with a learned sink per head and an output gate per head, over all earlier tokens or a sliding
window; optionally values blended with another layer's values of the same token.

   q, k, v = W_q h (+ b_q), W_k h (+ b_k), W_v h (+ b_v)       q, k of size key_dim per head, v of size value_dim
   v <- (1 - lambda) v + lambda v_first      (``value_mix`` "mixed"; "first": this layer's v is the v_first of the later
                                              layers; the blended v is what the cache keeps)
   the first ``position.rotary_dim`` numbers of every query and key head are rotated (position part: frequencies, pairs
   half-split or neighbours, a factor on cos and sin); the rest pass
   s[i, j] = scale * q_h[i] . k_g[j]     for j <= i, and i - j < window where there is a window
   p = exp(s) / (exp(sink_h) + sum_j exp(s))     the sink (``sink``) has no key and no value and is not scaled
   y = W_o concat_h(sigmoid(W_g h)_h * sum_j p[i, j] v_g[j]) (+ b_o)                          (``gate``)
Query head h reads kv head h // (num_heads / num_kv_heads).  Angles, scores, weights and sums are 32-bit in both
precisions.  The cache keeps pages of k and v.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from .. import native
from . import registry
from .base import ProjectedMixer
from .conv_attention import attend, rotation_options, window_plan
from .registry import register
from .spec import CacheEntry, CacheNeed, ParamSpec, PartSpec

FIRST_VALUES = "sink_attention.first_values"      # the name under which a step carries v_first


@register("mixer", "sink_attention")
class SinkAttention(ProjectedMixer):
    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, key_dim: int, value_dim: int, scale: float,
                 position: Optional[PartSpec] = None, window: Optional[int] = None, sink: bool = True, gate: bool = True,
                 qkv_bias: bool = False, out_bias: bool = False, value_mix: Optional[str] = None):
        if num_heads % num_kv_heads:
            raise ValueError("sink_attention: num_heads must be a multiple of num_kv_heads")
        if value_dim > 512 or key_dim > 4096:
            raise ValueError(f"sink_attention: sizes {key_dim} / {value_dim} are beyond what the kernels take (4096 / 512)")
        if value_mix not in (None, "first", "mixed"):
            raise ValueError(f"sink_attention: value_mix {value_mix!r} is not known")
        self.hidden_size, self.nh, self.nkv, self.dk, self.dv = hidden_size, num_heads, num_kv_heads, key_dim, value_dim
        self.scale = float(scale)
        # (a window beyond any context is one that never closes; the kernels take 32-bit sizes)
        self.window = min(int(window), 1 << 30) if window else None
        self.sink, self.gate, self.qkv_bias, self.out_bias, self.value_mix = sink, gate, qkv_bias, out_bias, value_mix
        self.position = registry.build("position", position) if position is not None else None
        if self.position is not None and not hasattr(self.position, "frequencies"):
            raise ValueError("sink_attention rotates by frequencies (a position part with ``frequencies``)")
        if self.position is not None and self.position.rotary_dim > key_dim:
            raise ValueError("sink_attention: rotary_dim exceeds key_dim")
        self.inner_cols = num_heads * value_dim

    def _qkv(self) -> Tuple[int, int, int]:
        return self.nh * self.dk, self.nkv * self.dk, self.nkv * self.dv

    def segments(self):
        s = {"qkv": self._qkv()}
        if self.gate:
            s["gate"] = (self.nh,)
        return s

    def inner_params(self) -> Dict[str, ParamSpec]:
        p = {}
        if self.qkv_bias:
            p["qkv.bias"] = ParamSpec((sum(self._qkv()),), role="vector", init="normal", rows=self._qkv())
        if self.sink:
            p["sink"] = ParamSpec((self.nh,), role="vector", init="normal")
        if self.value_mix:
            p["vmix"] = ParamSpec((1,), role="vector", init="half", rows=(1,), members_lack_axis=True)
        return p

    def cache_need(self) -> CacheNeed:
        return CacheNeed("pages", window=self.window,
                         entries=(CacheEntry("k", (self.nkv, self.dk)), CacheEntry("v", (self.nkv, self.dv))))

    def after_load(self) -> None:
        self._sink = self.w_sink.float().contiguous() if self.sink else None
        self._lambda = float(self.w_vmix.float().cpu()[0]) if self.value_mix == "mixed" else 0.0

    def launch_plan(self, step):
        return window_plan(step, self.nh, self.nkv, self.dk, self.dv, self.window, 0, self.rt.dtype)

    def inner(self, x, proj, step, cache, writes_cache, y, y_scale):
        T = y.shape[0]
        ws, dt = self.rt.workspace, self.rt.dtype
        nh, nkv, dk, dv = self.nh, self.nkv, self.dk, self.dv
        keep = first = None
        if self.value_mix == "first":
            keep = step.carried[FIRST_VALUES] = ws.get(FIRST_VALUES, (T, nkv * dv), dt)
        elif self.value_mix == "mixed":
            first = step.carried[FIRST_VALUES]
        pos = self.position
        freq = pos.frequencies(self.rt) if pos is not None and pos.rotary_dim else None
        q = ws.get("sa.q", (T, nh * dk), dt)
        native.conv_rope_write(q, proj["qkv"], nh, nkv, dk, dv, None, None, freq, pos.rotary_dim if freq is not None else 0,
                               step.positions, step.seq_of_token, step.cu_q, step.state_slots,
                               step.block_tables[cache.group], cache.page_size, cache.k_pages if writes_cache else None,
                               cache.v_pages if writes_cache else None, step.status,
                               bias=self.w_qkv_bias if self.qkv_bias else None, v_first=first, v_mix=self._lambda,
                               v_keep=keep, **rotation_options(pos))
        attend(self.launch_plan(step), ws, y, q, cache, step, nh, nkv, dk, dv, self.scale, 0.0, self.window, 0,
               sink=self._sink, gate=proj["gate"] if self.gate else None, out_scale=y_scale)
