"""Gated delta rule with a decay per key channel: a linear-attention mixer with a matrix state per head that forgets by
channel and writes only what it does not hold already (the delta rule of Yang et al. 2024, "Gated Delta Networks:
Improving Mamba2 with Delta Rule", with a decay for every key channel).

   q, k = W_q h, W_k h  (kv_heads x key_dim each),  v = W_v h  (heads x value_dim)
   q, k, v <- silu(conv(q, k, v))       causal, per channel, no bias, zeros before the request's start
   q <- q / sqrt(sum q^2 + 1e-6) * key_dim^(-1/2),   k <- k / sqrt(sum k^2 + 1e-6)          per head
   beta = sigmoid(W_b h) per head;   g = exp(-exp(A_log) softplus(W_a2 W_a1 h + dt_bias)) per head and key channel
   per head (head h reads q and k of h // (heads / kv_heads)), from S = 0:
       S <- diag(g_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t
   y = W_o (concat_h(rmsnorm(o_h; norm, eps)) * sigmoid(W_g2 W_g1 h))     the norm runs over one head's columns; its
                                                                         weight [value_dim] is shared by the heads
A request's state is S [heads, key_dim, value_dim] in 32-bit and the last taps - 1 rows that enter the convolution, both
in its state slot and zero at its first token.  The decays' inputs (the low-rank product hands them over in 32-bit), decays,
step sizes, unit norms, the recurrence and the output norm are 32-bit in both precisions.
"""
from __future__ import annotations

from typing import Dict

import torch

from .. import native
from .base import ProjectedMixer
from .linear import linear
from .registry import register
from .spec import CacheEntry, CacheNeed, ParamSpec

UNIT_EPS = 1e-6       # added to the sum of squares that a query or key is divided by


@register("mixer", "channel_delta_rule")
class ChannelDeltaRule(ProjectedMixer):
    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, key_dim: int, value_dim: int, taps: int,
                 decay_rank: int, gate_rank: int, norm_eps: float):
        if num_heads % num_kv_heads:
            raise ValueError("channel_delta_rule: num_heads must be a multiple of num_kv_heads")
        if not 1 <= key_dim <= 256:
            raise ValueError(f"channel_delta_rule: key_dim {key_dim} is beyond what the kernels take (1 to 256)")
        if not 1 <= taps <= 64:
            raise ValueError(f"channel_delta_rule: {taps} taps are beyond what the kernels take (1 to 64)")
        self.hidden_size, self.nh, self.nkv, self.dk, self.dv = hidden_size, num_heads, num_kv_heads, key_dim, value_dim
        self.taps, self.decay_rank, self.gate_rank, self.norm_eps = taps, decay_rank, gate_rank, float(norm_eps)
        self.inner_cols = num_heads * value_dim
        self._qkv = (num_kv_heads * key_dim, num_kv_heads * key_dim, num_heads * value_dim)
        self.channels = sum(self._qkv)

    def segments(self):
        return {"qkv": self._qkv, "a": (self.decay_rank,), "g": (self.gate_rank,), "b": (self.nh,)}

    def inner_params(self) -> Dict[str, ParamSpec]:
        return {"conv.weight": ParamSpec((self.channels, self.taps), role="vector", init="half", rows=self._qkv),
                "a2.weight": ParamSpec((self.nh * self.dk, self.decay_rank)),
                "g2.weight": ParamSpec((self.inner_cols, self.gate_rank)),
                "A_log": ParamSpec((self.nh,), role="vector", init="normal"),
                "dt_bias": ParamSpec((self.nh * self.dk,), role="vector", init="normal"),
                "norm": ParamSpec((self.dv,), role="vector", init="norm")}

    def cache_need(self) -> CacheNeed:
        states = (CacheEntry("S", (self.nh, self.dk, self.dv), "float32"),)
        if self.taps > 1:
            states += (CacheEntry("conv", (self.taps - 1, self.channels), "compute"),)
        return CacheNeed("state", states=states)

    def after_load(self) -> None:
        if self.w_A_log.dtype != self.w_dt_bias.dtype:       # (a checkpoint may hold one of them in 32-bit)
            self.w_A_log, self.w_dt_bias = self.w_A_log.float(), self.w_dt_bias.float()

    def inner(self, x, proj, step, cache, writes_cache, y, y_scale):
        T = y.shape[0]
        ws, dt = self.rt.workspace, self.rt.dtype
        H, G, dk, dv = self.nh, self.nkv, self.dk, self.dv
        f32 = torch.float32
        rows, conv = proj["qkv"], cache.states.get("conv")
        la = linear(proj["a"], self.w_a2_weight, None, ws.get("dr.la", (T, H * dk), f32))
        gate = linear(proj["g"], self.w_g2_weight, None, ws.get("dr.gate", (T, H * dv), dt))
        if step.max_q_len == 1 and T == step.num_seqs and not step.plan_for_any_batch and native.delta_step_supports(dk, dv):
            # (every request brings one row: the rest is one kernel)
            native.delta_step(y, rows, self.w_conv_weight, conv, la, self.w_A_log, self.w_dt_bias, proj["b"], gate, self.w_norm,
                              self.norm_eps, y_scale, cache.states["S"], step.cu_q, step.state_slots, step.num_seqs, G, H, dk,
                              dv, dk ** -0.5, UNIT_EPS, writes_cache)
            if conv is not None and writes_cache and G != H:
                native.conv_state_update(conv, rows, step.cu_q, step.state_slots, step.num_seqs)
            return
        u = ws.get("dr.u", (T, self.channels), dt)
        rn = ws.get("dr.rn", (T, 2 * G), f32)
        beta = ws.get("dr.beta", (T, H), f32)
        native.delta_prepare(u, rn, rows, self.w_conv_weight, conv, la, self.w_A_log, self.w_dt_bias, proj["b"], beta,
                             step.seq_of_token, step.cu_q, step.state_slots, G, H, dk, dv, dk ** -0.5, UNIT_EPS)
        if conv is not None and writes_cache:
            native.conv_state_update(conv, rows, step.cu_q, step.state_slots, step.num_seqs)
        o = ws.get("dr.o", (T, H * dv), f32)
        n = native.delta_scratch_elems(T, step.num_seqs, H, dk, dv, dt, step.max_q_len)
        native.delta_scan(o, u, rn, la, beta, cache.states["S"], step.cu_q, step.state_slots, step.num_seqs, G, H, dk, dv,
                          writes_cache, scratch=ws.get("dr.chunks", (n,), f32) if n else None, max_q_len=step.max_q_len)
        native.gla_gate_norm(y, o, gate, self.w_norm, self.norm_eps, H, dv, step.seq_of_token, "sigmoid", y_scale)
