"""Grouped-query attention behind a short causal convolution, with capped scores and a sliding window that always
keeps a request's first tokens.

   [q | k | v] = x W_qkv^T;  q_h, k_g of size key_dim, v_g of size value_dim (they may differ)
   every channel c of q, k and v is convolved over time:  y_t[c] = sum_j w[c, j] * u_(t - taps + 1 + j)[c]
       (zeros before the request's first token; the request's last taps - 1 projected rows are its state)
   the first rotary_dim numbers of every query and key head are rotated by position * frequency,
       pairs (i, i + rotary_dim / 2); the rest pass
   s[i, j] = scale * q_h[i] . k_g[j];   s <- softcap * tanh(s / softcap)
   position i sees j if j <= i and (i - j < window or j < keep_first); kept tokens keep their positions
   o_h[i] = softmax_j(s[i, j]) v_g[j];   y = concat_h(o_h) W_o^T
Query head h reads kv head h // (num_heads / num_kv_heads).  Convolution, window, kept tokens, cap and rotation are
each an option of the constructor.  The convolution's sums, angles, scores, weights and sums are 32-bit in both
precisions.  The cache keeps pages of k and v (the pages of the first keep_first positions are never given back)
and, with a convolution, the state array ``conv`` [taps - 1, channels].
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import native
from . import registry
from .base import Mixer
from .linear import PendingProduct, linear, may_defer
from .registry import register
from .spec import CacheEntry, CacheNeed, ParamSpec, PartSpec


def rotation_options(position) -> dict:
    """What ``native.conv_rope_write`` has to know of a position part that gives frequencies."""
    if position is None:
        return {}
    return {"neighbours": getattr(position, "neighbours", False), "magnitude": getattr(position, "magnitude", 1.0)}


def window_plan(step, nh: int, nkv: int, dk: int, dv: int, window: Optional[int], keep_first: int, dtype, maps: int = 1):
    """(into how many shares the tensor-core kernel cuts the key tiles of every unit, or 0 for the plain kernel;
    whether a unit is a token with the query heads of one key head as rows, which steps of single tokens use, or
    a tile of 64 tokens with one head), for attention over a window that keeps first tokens (or over all keys); maps:
    attention maps per head."""
    key = ("window_attention", nh, nkv, dk, dv, window or 0, keep_first, maps)
    plan = step.plans.get(key)
    if plan is None:
        if native.WINDOW_TC and native.window_attention_tc_supports(dk, dv, dtype, maps):
            longest = min(step.max_ctx_len, window + keep_first) if window else step.max_ctx_len
            heads_rows = step.max_q_len <= 1 and nh // nkv <= native.WINDOW_TC_ROWS
            if heads_rows:
                units = step.num_tokens * nkv
            elif step.max_q_len <= 1:
                units = step.num_tokens * nh
            else:
                units = (-(-step.num_tokens // native.WINDOW_TC_ROWS) + step.num_seqs - 1) * nh
            # (two CTAs of one map fit an SM, one of two maps; steps with prompt portions fill it once before their keys
            # are shared out: the shares cost a pass over 32-bit partial outputs of every row)
            if step.max_q_len <= 1 and maps > 1:      # (one CTA to an SM: no second round)
                nsplit = max(1, min(native.SM_COUNT // max(units, 1), -(-longest // 128), 64))
            else:
                nsplit = native.attention_mixed_splits(units, longest, per_sm=2 if step.max_q_len <= 1 else 1, min_share=128)
            plan = (nsplit, heads_rows)
        else:
            plan = (0, False)
        step.plans[key] = plan
    return plan


def attend(plan, ws, o, q, cache, step, nh: int, nkv: int, dk: int, dv: int, scale: float, softcap: float,
           window: Optional[int], keep_first: int, **extras) -> None:
    """Runs the attention of ``plan`` (``window_plan``) over the cache's pages; extras: sink, gate, out_scale, chunked,
    maps (lambda, eps)."""
    bt = step.block_tables[cache.group]
    nsplit, heads_rows = plan
    if nsplit:
        scratch = None
        if nsplit > 1:
            scratch = ws.get("cwa.splits", (native.attention_mixed_scratch_elems(q.shape[0], nh * (2 if extras.get("maps") else 1), dv, nsplit),), torch.float32)
        native.window_attention_tc(o, q, cache.k_pages, cache.v_pages, bt, step.positions, step.seq_of_token,
                                   step.cu_q, step.num_seqs, nh, nkv, dk, dv, scale, softcap, window or 0, keep_first,
                                   nsplit, scratch, heads_rows, **extras)
    else:
        native.window_attention(o, q, cache.k_pages, cache.v_pages, bt, step.positions, step.seq_of_token, nh, nkv,
                                dk, dv, scale, softcap, window or 0, keep_first, **extras)


@register("mixer", "conv_window_attention")
class ConvWindowAttention(Mixer):
    graph_safe = True
    takes_scaled_rows = True      # x may be ScaledRows: the qkv product finishes the norm
    defers_output = True          # forward(..., defer=True) may hand the output projection on unrun

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, key_dim: int, value_dim: int, scale: float,
                 softcap: Optional[float] = None, taps: Optional[int] = None, position: Optional[PartSpec] = None,
                 window: Optional[int] = None, keep_first: int = 0):
        if num_heads % num_kv_heads:
            raise ValueError("num_heads must be a multiple of num_kv_heads")
        if taps is not None and not 1 <= taps <= 64:
            raise ValueError(f"conv_window_attention: {taps} taps are beyond what the kernel takes (1 to 64)")
        if value_dim > 512:
            raise ValueError(f"conv_window_attention: value_dim {value_dim} is beyond what the kernels take (512)")
        self.hidden_size, self.nh, self.nkv, self.dk, self.dv = hidden_size, num_heads, num_kv_heads, key_dim, value_dim
        self.scale, self.softcap, self.taps = float(scale), (float(softcap) if softcap else 0.0), taps
        # (a window beyond any context is one that never closes; the kernels take 32-bit sizes)
        self.window = min(int(window), 1 << 30) if window else None
        self.keep_first = min(int(keep_first), 1 << 30) if window else 0
        self.position = registry.build("position", position) if position is not None else None
        if self.position is not None and not hasattr(self.position, "frequencies"):
            raise ValueError("conv_window_attention rotates by frequencies (a position part with ``frequencies``)")
        if self.position is not None and self.position.rotary_dim > key_dim:
            raise ValueError("rotary_dim exceeds key_dim")
        self.channels = (num_heads + num_kv_heads) * key_dim + num_kv_heads * value_dim

    def params(self) -> Dict[str, ParamSpec]:
        q, k, v = self.nh * self.dk, self.nkv * self.dk, self.nkv * self.dv
        p = {"qkv.weight": ParamSpec((q + k + v, self.hidden_size), rows=(q, k, v)),
             "o.weight": ParamSpec((self.hidden_size, self.nh * self.dv))}
        if self.taps is not None:
            p["conv.weight"] = ParamSpec((q + k + v, self.taps), role="vector", init="half", rows=(q, k, v))
        return p

    def cache_need(self) -> CacheNeed:
        states = ()
        if self.taps is not None and self.taps > 1:
            states = (CacheEntry("conv", (self.taps - 1, self.channels), "compute"),)
        return CacheNeed("pages", window=self.window, keep_first=self.keep_first,
                         entries=(CacheEntry("k", (self.nkv, self.dk)), CacheEntry("v", (self.nkv, self.dv))),
                         states=states)

    def launch_plan(self, step):
        """(into how many shares the tensor-core kernel cuts the key tiles of every unit, or 0 for the plain kernel;
        whether a unit is a token with the query heads of one key head as rows, which steps of single tokens use, or
        a tile of 64 tokens with one head).  Where the units do not fill the device (decoding, short portions) their
        keys are shared out, in shares of at least 128."""
        return window_plan(step, self.nh, self.nkv, self.dk, self.dv, self.window, self.keep_first, self.rt.dtype)

    def forward(self, x, step, cache, writes_cache, defer=False):
        T = x.shape[0]
        ws, dt = self.rt.workspace, self.rt.dtype
        nh, nkv, dk, dv = self.nh, self.nkv, self.dk, self.dv
        qkv = linear(x, self.w_qkv_weight, None, ws.get("cwa.qkv", (T, self.channels), dt))
        bt = step.block_tables[cache.group]
        conv_w = self.w_conv_weight if self.taps is not None else None
        conv_state = cache.states.get("conv")
        freq = self.position.frequencies(self.rt) if self.position is not None else None
        q = ws.get("cwa.q", (T, nh * dk), dt)
        native.conv_rope_write(q, qkv, nh, nkv, dk, dv, conv_w, conv_state, freq,
                               self.position.rotary_dim if self.position is not None else 0, step.positions,
                               step.seq_of_token, step.cu_q, step.state_slots, bt, cache.page_size,
                               cache.k_pages if writes_cache else None, cache.v_pages if writes_cache else None,
                               step.status, **rotation_options(self.position))
        if conv_state is not None and writes_cache:
            native.conv_state_update(conv_state, qkv, step.cu_q, step.state_slots, step.num_seqs)
        o = ws.get("cwa.o", (T, nh * dv), dt)
        attend(self.launch_plan(step), ws, o, q, cache, step, nh, nkv, dk, dv, self.scale, self.softcap, self.window,
               self.keep_first)
        out = ws.get("cwa.out", (T, self.hidden_size), dt)
        if defer and may_defer(o, self.w_o_weight):
            return PendingProduct(o, self.w_o_weight, None, out)
        return linear(o, self.w_o_weight, None, out)
