"""Routed experts: a mixture of small gated feed-forwards of which every row uses ``top``.

   z = W_router x  (32-bit);   score = sigmoid(z)  or  softmax(z)            ``score``
   the ``top`` experts with the largest choice scores are chosen (ties: the lower index); a choice score is the score,
       plus a number per expert with ``correction``; with ``groups`` (count, keep) the experts form ``count`` groups of
       neighbours and only those in the ``keep`` groups with the largest choice score can be chosen
   their weights are their scores (without the correction), divided by their sum (+ ``sum_eps``) if ``renormalize``,
       times ``factor``
   expert e:  f_e(h) = W_down,e (silu(W_gate,e h) * (W_up,e h)),  or with ``limit`` the clamped form
       g = min(W_gate,e h, limit), u = clamp(W_up,e h, -limit, limit):  W_down,e (g sigmoid(1.702 g) (u + 1))
   the last ``identity`` of the router's num_experts + identity outputs are identity experts:  f_e(h) = h, without tensors
   y = sum over the chosen e of  f_e(w_e * x)   (``weight_on`` "input")   or   w_e * f_e(x)   ("output")
   with a shared expert of ``shared_size``:  y += sigmoid(w_sg . x) * f_shared(x)   (``shared_gate``; without it the
       shared expert is added as it is); its own limit is ``shared_limit``
Router logits, scores, weights and the gate are 32-bit in both precisions.  Rows are sorted by expert on the device
(no host round trip: the launches depend on the step's shape alone), every expert's rows run as tiles of one grouped
product, and a row's choices are added up in a fixed order.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from .. import native
from .base import FeedForward
from .linear import gated_linear, linear
from .registry import register
from .spec import ParamSpec


@register("ffn", "routed_experts")
class RoutedExperts(FeedForward):
    graph_safe = True

    def __init__(self, hidden_size: int, num_experts: int, top: int, intermediate_size: int,
                 shared_size: Optional[int] = None, score: str = "sigmoid", renormalize: bool = False,
                 weight_on: str = "input", shared_gate: bool = False, correction: bool = False,
                 groups: Optional[Tuple[int, int]] = None, identity: int = 0, factor: float = 1.0, sum_eps: float = 0.0,
                 limit: Optional[float] = None, shared_limit: Optional[float] = None):
        if score not in ("sigmoid", "softmax") or weight_on not in ("input", "output"):
            raise ValueError(f"routed_experts: score {score!r} / weight_on {weight_on!r} not known")
        outputs = num_experts + identity
        if groups and (groups[0] < 1 or outputs % groups[0] or not 1 <= groups[1] <= groups[0]
                       or top > groups[1] * (outputs // groups[0])):
            raise ValueError(f"routed_experts: {groups[1]} of {groups[0]} groups of {outputs} experts do not give {top} to choose")
        if identity and weight_on == "input":
            raise ValueError("routed_experts: identity experts take their weight on the output")
        if not 1 <= top <= min(outputs, 32) or outputs > 1024:
            raise ValueError(f"routed_experts: top {top} of {num_experts} experts is beyond what the kernels take")
        self.hidden_size, self.E, self.top, self.ff = hidden_size, num_experts, top, intermediate_size
        self.shared_size = shared_size or None
        self.score, self.renormalize, self.weight_on = score, bool(renormalize), weight_on
        self.shared_gate = bool(shared_gate) and self.shared_size is not None
        self.correction, self.groups, self.identity = bool(correction), groups or (1, 1), int(identity)
        self.factor, self.sum_eps = float(factor), float(sum_eps)
        self.act, self.limit = ("silu", 0.0) if limit is None else ("clamped", float(limit))
        self.shared_act, self.shared_limit = ("silu", 0.0) if shared_limit is None else ("clamped", float(shared_limit))

    def params(self) -> Dict[str, ParamSpec]:
        H, E, F = self.hidden_size, self.E, self.ff
        outputs = E + self.identity
        rows = (outputs, 1) if self.shared_gate else (outputs,)
        pad = -sum(rows) % 8                     # (the product's width in steps of 8)
        p = {"router.weight": ParamSpec((sum(rows) + pad, H), rows=rows, pad=pad),
             "gate_up.weight": ParamSpec((E * 2 * F, H), rows=(F,) * (2 * E)),
             "down.weight": ParamSpec((E * H, F), rows=(H,) * E)}
        if self.correction:
            p["correction"] = ParamSpec((outputs,), role="vector", init="normal")
        if self.shared_size is not None:
            S = self.shared_size
            p["shared.gate_up.weight"] = ParamSpec((2 * S, H), rows=(S, S))
            p["shared.down.weight"] = ParamSpec((H, S))
        return p

    def forward(self, x, step):
        T, H = x.shape
        E, top, F = self.E, self.top, self.ff
        ws, dt = self.rt.workspace, self.rt.dtype
        R = T * top
        n_logits = self.w_router_weight.shape[0]
        logits = linear(x, self.w_router_weight, None, ws.get("moe.logits", (T, n_logits), torch.float32))
        ids = ws.get("moe.ids", (T, top), torch.int32)
        wts = ws.get("moe.wts", (T, top), torch.float32)
        counts = ws.get("moe.counts", (1024,), torch.int32, zero=True)     # zero between steps: moe_place leaves it so
        native.moe_route(logits, E + self.identity, top, self.score, self.renormalize, step.seq_of_token, ids, wts, counts,
                         self.identity, self.sum_eps, self.factor, self.w_correction if self.correction else None,
                         *self.groups)
        offsets = ws.get("moe.offsets", (E + 1,), torch.int32)
        row_token = ws.get("moe.row_token", (R,), torch.int32)
        row_w = ws.get("moe.row_w", (R,), torch.float32)
        pair_pos = ws.get("moe.pair_pos", (R,), torch.int32)
        native.moe_place(ids, wts, E, counts, offsets, row_token, row_w, pair_pos)
        on_input = self.weight_on == "input"
        act = ws.get("moe.act", (R, F), dt)
        y = ws.get("moe.y", (R, H), dt)
        w_in, w_out, weight = self.w_gate_up_weight.view(E, 2 * F, H), self.w_down_weight.view(E, H, F), row_w if on_input else None
        if native.moe_pairs_pay(R, E, F, H, dt) and native.moe_pairs_pay(R, E, H, F, dt) and x.stride(0) % 8 == 0:
            rows = ws.get("moe.rows", (R, H), dt)          # long portions: every expert's rows gathered, then tcgen05
            native.moe_gather(rows, x, offsets, E, row_token, weight)
            native.gemm_pairs_grouped(rows, w_in, act, offsets, gated=True, act=self.act, limit=self.limit)
            native.gemm_pairs_grouped(act, w_out, y, offsets)
        else:
            native.moe_gemm(act, x, w_in, offsets, gated=True, row_token=row_token, row_w=weight, act=self.act,
                            limit=self.limit)
            native.moe_gemm(y, act, w_out, offsets)
        shared = None
        if self.shared_size is not None:
            S = self.shared_size
            f = gated_linear(x, self.w_shared_gate_up_weight, ws.get("moe.shared.act", (T, S), dt),
                             lambda m, n: ws.get("moe.shared.gate_up", (m, n), dt), self.shared_act, self.shared_limit)
            shared = linear(f, self.w_shared_down_weight, None, ws.get("moe.shared.out", (T, H), dt))
        out = ws.get("moe.out", (T, H), dt)
        native.moe_combine(out, y, pair_pos, top, None if on_input else wts, shared,
                           logits[:, E + self.identity:E + self.identity + 1] if self.shared_gate else None, step.seq_of_token,
                           x if self.identity else None, ids if self.identity else None, E)
        return out
