"""A plain, slow implementation of the Vunepel design in float64 on the CPU: one function per mechanism, whole
sequences at once, no cache, no state carried between calls.  It shares no code with the package; the tests compare
the engine with it.

A model is (config dict as in config.json, {tensor name: float64 tensor}).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F = torch.float64


def dynamic_tanh(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, alpha: torch.Tensor) -> torch.Tensor:
    return torch.tanh(alpha * x) * w + b


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def causal_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [T, C], w [C, taps]: sum_j w[:, j] u_(t - taps + 1 + j), zeros before the first row."""
    T, C = u.shape
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=u.dtype), u], 0)
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + padded[j:j + T] * w[:, j]
    return y


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def channel_decays(z: torch.Tensor, A_log: torch.Tensor, dt_bias: torch.Tensor) -> torch.Tensor:
    """z, dt_bias [.., H, d]; A_log [H] -> the factor of every key channel, in (0, 1)."""
    return torch.exp(-torch.exp(A_log)[:, None] * torch.nn.functional.softplus(z + dt_bias, threshold=1e9))


def delta_rule(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor) -> torch.Tensor:
    """q, k, g [T, H, d], v [T, H, dv], beta [T, H]: per head and token, from a state of zeros,
    S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    o = torch.zeros_like(v)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return o


def channel_delta(h: torch.Tensor, P: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ P[n].T, P[n + ".conv"])) for n in ("q", "k", "v"))
    q = unit(q.view(T, G, d)).repeat_interleave(H // G, dim=1) * d ** -0.5
    k = unit(k.view(T, G, d)).repeat_interleave(H // G, dim=1)
    g = channel_decays(((h @ P["a1"].T) @ P["a2"].T).view(T, H, d), P["A_log"], P["dt_bias"].view(H, d))
    o = delta_rule(q, k, v.view(T, H, dv), g, torch.sigmoid(h @ P["b"].T))
    o = (rms(o, eps) * P["norm"]).reshape(T, H * dv)
    return (o * torch.sigmoid((h @ P["g1"].T) @ P["g2"].T)) @ P["o"].T


def rotate_halves(x: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [T, heads, d]: the first rot.dims numbers of a head are turned by the row's position, pair (i, i + dims/2)."""
    if not rot or not rot["dims"]:
        return x
    dims = rot["dims"]
    half = dims // 2
    f = torch.tensor([rot["base"] ** (-2.0 * i / dims) for i in range(half)], dtype=F)
    ang = torch.arange(x.shape[0], dtype=F)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], dim=-1)


def visible(T: int, chunk: Optional[int]) -> torch.Tensor:
    """Earlier tokens of the same chunk (chunks of ``chunk`` positions from the sequence's first)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen if chunk is None else seen & (i // chunk == j // chunk)


def softmax_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, chunk: Optional[int]) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]."""
    T, H = q.shape[:2]
    per = H // k.shape[1]
    k, v = k.repeat_interleave(per, dim=1), v.repeat_interleave(per, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(~visible(T, chunk)[None], -math.inf)
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, dim=-1), v)


def two_map_weight(P: Dict[str, torch.Tensor], diff: float) -> torch.Tensor:
    return torch.exp((P["lq1"] * P["lk1"]).sum()) - torch.exp((P["lq2"] * P["lk2"]).sum()) + diff


def keys_and_values(h: torch.Tensor, P: Dict[str, torch.Tensor], m: dict, eps: float):
    """(keys [T, G, 2, d] normed and rotated, values [T, G, dv]) of an attention layer with projections of its own."""
    T = h.shape[0]
    G, d, dv = m["kv_heads"], m["dim"], m["vdim"]
    k = rms((h @ P["k"].T).view(T, 2 * G, d), eps) * P["k.norm"]
    return rotate_halves(k, m.get("rot")).view(T, G, 2, d), (h @ P["v"].T).view(T, G, dv)


def differential_attention(h: torch.Tensor, P: Dict[str, torch.Tensor], m: dict, eps: float, kv) -> torch.Tensor:
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    k, v = kv
    q = rms((h @ P["q"].T).view(T, 2 * H, d), eps) * P["q.norm"]
    q = rotate_halves(q, m.get("rot")).view(T, H, 2, d)
    chunk = m["mask"]["size"] if m.get("mask") else None
    a1, a2 = (softmax_attention(q[:, :, i], k[:, :, i], v, m["scale"], chunk) for i in (0, 1))
    o = rms(a1 - two_map_weight(P, m["diff"]) * a2, eps) * (1.0 - m["diff"])
    return o.reshape(T, H * dv) @ P["o"].T


def part(W: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}


def clamped_mlp(h: torch.Tensor, P: Dict[str, torch.Tensor], prefix: str, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ P[prefix + "gate"].T, max=limit)
    u = torch.clamp(h @ P[prefix + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ P[prefix + "down"].T


def choose(s: torch.Tensor, top: int) -> List[int]:
    return torch.topk(s, top).indices.tolist()


def expert_mixture(h: torch.Tensor, P: Dict[str, torch.Tensor], mlp: dict) -> torch.Tensor:
    r = mlp["router"]
    s = torch.sigmoid(h @ P["router"].T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids = choose(s[t], r["top"])
        w = s[t, ids] / (s[t, ids].sum() + 1e-20) * r["scale"]
        for e, we in zip(ids, w):
            out[t] += we * clamped_mlp(h[t:t + 1], P, f"e{e}.", mlp["expert"]["limit"])[0]
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ P["shared.sg"].T) * clamped_mlp(h, P, "shared.", mlp["shared"]["limit"])
    return out


def feed_forward(h: torch.Tensor, P: Dict[str, torch.Tensor], mlp: dict) -> torch.Tensor:
    return clamped_mlp(h, P, "", mlp["limit"]) if mlp["kind"] == "dense" else expert_mixture(h, P, mlp)


def forward(cfg: dict, W: Dict[str, torch.Tensor], tokens, return_layers: bool = False):
    """Logits [T, vocab] of one whole sequence (and the residual stream after every layer)."""
    eps = cfg["norm"]["eps"]
    norm = lambda x, n: dynamic_tanh(x, W[n], W[n + ".b"], W[n + ".alpha"])
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    streams, kept = [], {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h, mix = norm(x, p + "norm1"), part(W, p + "mix.")
        if L["type"] == "channel_delta":
            y = channel_delta(h, mix, m, eps)
        else:
            if m.get("kv_from") is None:
                kept[i] = keys_and_values(h, mix, m, eps)
            y = differential_attention(h, mix, m, eps, kept[i if m.get("kv_from") is None else m["kv_from"]])
        if L.get("mlp"):
            y = y + feed_forward(h, part(W, p + "mlp."), L["mlp"])
        x = x + y
        streams.append(x)
    logits = norm(x, "final.norm") @ W["head"].T
    return (logits, torch.stack(streams)) if return_layers else logits
