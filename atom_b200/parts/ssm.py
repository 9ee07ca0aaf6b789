"""State-space duality (Mamba-2, Dao and Gu 2024): a matrix state per head with one decay per head and token.

   [z | x | B | C | dt] = W_in h          inner = heads * value_dim numbers of z and x, groups * state of B and C, heads of dt
   x, B, C <- silu(conv(x, B, C) + b)     causal, per channel, zeros before the request's start
   dt <- softplus(dt + dt_bias)
   per head (head h reads B and C of group h // (heads / groups)):
       S_t = exp(-exp(A_log) dt) S_(t-1) + dt B_t x_t^T,   y_t = S_t^T C_t + D x_t         S = 0 before the first token
   y <- y * silu(z), RMS-normed in ``norm_groups`` equal parts, times a weight;   out = W_o y
A request's state is S [heads, state, value_dim] in 32-bit and the last taps - 1 rows that enter the convolution, both
in its state slot and zero at its first token.  dt, decays, the recurrence, the gate and the norm are 32-bit in both
precisions.
"""
from __future__ import annotations

from typing import Dict

import torch

from .. import native
from .base import ProjectedMixer
from .registry import register
from .spec import CacheEntry, CacheNeed, ParamSpec


@register("mixer", "state_space")
class StateSpace(ProjectedMixer):
    def __init__(self, hidden_size: int, num_heads: int, value_dim: int, state_dim: int, groups: int, taps: int,
                 norm_groups: int, norm_eps: float):
        if num_heads % groups:
            raise ValueError(f"state_space: {num_heads} heads are no multiple of {groups} groups")
        if (num_heads * value_dim) % norm_groups:
            raise ValueError(f"state_space: {num_heads * value_dim} numbers do not make {norm_groups} equal parts")
        if not 1 <= state_dim <= 256:
            raise ValueError(f"state_space: state size {state_dim} is beyond what the kernel takes (1 to 256)")
        if not 1 <= taps <= 64:
            raise ValueError(f"state_space: {taps} taps are beyond what the kernels take (1 to 64)")
        self.hidden_size, self.nh, self.dv, self.n, self.g = hidden_size, num_heads, value_dim, state_dim, groups
        self.taps, self.norm_groups, self.norm_eps = taps, norm_groups, float(norm_eps)
        self.inner_cols = num_heads * value_dim
        self.channels = self.inner_cols + 2 * groups * state_dim

    def segments(self):
        return {"in": (self.inner_cols + self.channels + self.nh,)}

    def inner_params(self) -> Dict[str, ParamSpec]:
        return {"conv.weight": ParamSpec((self.channels, self.taps), role="vector", init="half"),
                "conv.bias": ParamSpec((self.channels,), role="vector", init="normal"),
                "dt_bias": ParamSpec((self.nh,), role="vector", init="normal"),
                "A_log": ParamSpec((self.nh,), role="vector", init="normal"),
                "D": ParamSpec((self.nh,), role="vector", init="norm"),
                "norm": ParamSpec((self.inner_cols,), role="vector", init="norm")}

    def cache_need(self) -> CacheNeed:
        states = (CacheEntry("S", (self.nh, self.n, self.dv), "float32"),)
        if self.taps > 1:
            states += (CacheEntry("conv", (self.taps - 1, self.channels), "compute"),)
        return CacheNeed("state", states=states)

    def after_load(self) -> None:
        self._D = self.w_D.float().contiguous()

    def inner(self, x, proj, step, cache, writes_cache, y, y_scale):
        T = y.shape[0]
        ws, dt_ = self.rt.workspace, self.rt.dtype
        H, P, N, G, I, C = self.nh, self.dv, self.n, self.g, self.inner_cols, self.channels
        rows = proj["in"]
        u = ws.get("ssm.u", (T, C), dt_)
        dt = ws.get("ssm.dt", (T, H), torch.float32)
        la = ws.get("ssm.la", (T, H), torch.float32)
        native.ssm_conv(u, rows[:, I:I + C], self.w_conv_weight, self.w_conv_bias, cache.states.get("conv"), dt, la,
                        rows[:, I + C:], self.w_dt_bias, self.w_A_log, step.seq_of_token, step.cu_q, step.state_slots,
                        step.num_seqs, writes_cache)
        o = ws.get("ssm.o", (T, I), torch.float32)
        run, _ = native.ssm_run(min(T, step.max_q_len), N, P, dt_)
        nb, na = native.ssm_scratch_elems(T, step.num_seqs, H, N, P, run)
        sb = ws.get("ssm.runs", (nb,), torch.float32) if nb else None
        sa = ws.get("ssm.run_decays", (na,), torch.float32) if na else None
        native.ssm_scan(o, u, dt, la, self._D, cache.states["S"], sb, sa, step.cu_q, step.state_slots, step.num_seqs,
                        H, G, N, P, writes_cache, step.max_q_len)
        native.ssm_gate_norm(y, o, rows[:, :I], self.w_norm, self.norm_groups, self.norm_eps, y_scale, step.seq_of_token)
