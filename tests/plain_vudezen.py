"""A plain, slow implementation of the Vudezen design in float64 on the CPU: one function per mechanism, whole
sequences at once, no cache, no state carried between calls.  It shares no code with the package; the tests compare
the engine with it.

A model is (config dict as in config.json, {tensor name: float64 tensor}).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

F = torch.float64


def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    mean = x.mean(-1, keepdim=True)
    var = ((x - mean) ** 2).mean(-1, keepdim=True)
    return (x - mean) / torch.sqrt(var + eps) * w + b


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def pair_frequencies(rot: dict) -> Tuple[torch.Tensor, float]:
    """(frequency of every pair, factor on cos and sin); YaRN's stretch where ``scaling`` is given."""
    d, base = rot["dims"], rot["base"]
    f = torch.tensor([base ** (-2.0 * i / d) for i in range(d // 2)], dtype=F)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    turns = lambda t: d * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(turns(sc["fast"])), 0), min(math.ceil(turns(sc["slow"])), d - 1)
    ramp = torch.clamp((torch.arange(d // 2, dtype=F) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate_neighbours(x: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [T, heads, d]: numbers 2i and 2i + 1 of the first ``rot.dims`` are turned by position * frequency_i."""
    if not rot or rot["dims"] == 0:
        return x
    T, d = x.shape[0], rot["dims"]
    f, mag = pair_frequencies(rot)
    ang = torch.arange(T, dtype=F)[:, None] * f[None, :]
    c, s = (torch.cos(ang) * mag)[:, None, :], (torch.sin(ang) * mag)[:, None, :]
    y = x.clone()
    u, v = x[..., 0:d:2], x[..., 1:d:2]
    y[..., 0:d:2] = u * c - v * s
    y[..., 1:d:2] = v * c + u * s
    return y


def visible(T: int, size: Optional[int]) -> torch.Tensor:
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen if size is None else seen & (i - j < size)


def sink_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, sink: torch.Tensor,
                   window: Optional[int]) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]: weights exp(s) / (exp(sink_h) + sum exp(s))."""
    T, H = q.shape[:2]
    per = H // k.shape[1]
    k, v = k.repeat_interleave(per, dim=1), v.repeat_interleave(per, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(~visible(T, window)[None], -math.inf)
    s = torch.cat([s, sink[:, None, None].expand(H, T, 1)], dim=-1)
    w = torch.softmax(s, dim=-1)[..., :T]                  # (the sink takes a share and has no value)
    return torch.einsum("hij,jhd->ihd", w, v)


def attention(h: torch.Tensor, P: Dict[str, torch.Tensor], m: dict, v_first: Optional[torch.Tensor] = None):
    """The attention mixer on h [T, width]; P holds q, k, v, o, g, sink and biases as ``<name>.b``.  v_first: another
    layer's values of the same tokens, mixed in with P['vmix'].  Returns (output, this layer's values)."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    lin = lambda n, x: x @ P[n].T + (P[n + ".b"] if n + ".b" in P else 0.0)
    q, k, v = lin("q", h).view(T, H, d), lin("k", h).view(T, G, d), lin("v", h).view(T, G, dv)
    if v_first is not None:
        v = (1.0 - P["vmix"]) * v + P["vmix"] * v_first
    rot = m.get("rot")
    window = m["mask"]["size"] if m.get("mask") else None
    o = sink_attention(rotate_neighbours(q, rot), rotate_neighbours(k, rot), v, m["scale"], P["sink"], window)
    o = o * torch.sigmoid(h @ P["g"].T)[:, :, None]
    return lin("o", o.reshape(T, H * dv)), v


def biased_conv(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """u [T, C], w [C, taps], b [C]: sum_j w[:, j] u_(t - taps + 1 + j) + b, zeros before the first row."""
    T, C = u.shape
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=u.dtype), u], 0)
    y = b.expand(T, C).clone()
    for j in range(taps):
        y = y + padded[j:j + T] * w[:, j]
    return y


def state_space(x: torch.Tensor, B: torch.Tensor, C: torch.Tensor, dt: torch.Tensor, A_log: torch.Tensor,
                D: torch.Tensor) -> torch.Tensor:
    """x [T, H, P], B and C [T, groups, N], dt [T, H] (after softplus), token by token from a state of zeros:
    S_t = exp(-exp(A_log) dt) S_(t-1) + dt B_t x_t^T;  y_t = S_t^T C_t + D x_t."""
    T, H, Pd = x.shape
    per = H // B.shape[1]
    B, C = B.repeat_interleave(per, dim=1), C.repeat_interleave(per, dim=1)
    S = torch.zeros(H, B.shape[2], Pd, dtype=x.dtype)
    y = torch.zeros_like(x)
    for t in range(T):
        a = torch.exp(-torch.exp(A_log) * dt[t])
        S = a[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnp,hn->hp", S, C[t]) + D[:, None] * x[t]
    return y


def grouped_rms_norm(y: torch.Tensor, w: torch.Tensor, parts: int, eps: float) -> torch.Tensor:
    T, n = y.shape
    z = y.view(T, parts, n // parts)
    return (z / torch.sqrt((z * z).mean(-1, keepdim=True) + eps)).reshape(T, n) * w


def mamba2(h: torch.Tensor, P: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, Pd, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * Pd
    z, xbc, dt = torch.split(h @ P["in"].T, [inner, inner + 2 * G * N, H], dim=1)
    xbc = silu(biased_conv(xbc, P["conv"], P["conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=1)
    dt = torch.nn.functional.softplus(dt + P["dt_bias"], threshold=1e9)
    y = state_space(x.view(T, H, Pd), B.reshape(T, G, N), C.reshape(T, G, N), dt, P["A_log"], P["D"]).reshape(T, inner)
    return grouped_rms_norm(y * silu(z), P["norm"], m["norm_groups"], eps) @ P["o"].T


def part(W: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}


def two_mixers(h: torch.Tensor, P: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    left, _ = attention(h, part(P, "left."), m["left"])
    return m["left_scale"] * left + m["right_scale"] * mamba2(h, part(P, "right."), m["right"], eps)


def clamped_expert(h: torch.Tensor, P: Dict[str, torch.Tensor], prefix: str, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ P[prefix + "gate"].T, max=limit)
    u = torch.clamp(h @ P[prefix + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ P[prefix + "down"].T


def choose(s: torch.Tensor, correction: torch.Tensor, router: dict) -> List[int]:
    """The experts of one token with scores s [n]."""
    c = s + correction
    n = c.shape[0]
    groups = router.get("groups")
    if groups:
        size = n // groups["count"]
        best = torch.topk(c.view(groups["count"], size).max(dim=1).values, groups["keep"]).indices.tolist()
        barred = torch.tensor([i // size not in best for i in range(n)])
        c = c.masked_fill(barred, -math.inf)
    return torch.topk(c, router["top"]).indices.tolist()


def expert_mixture(h: torch.Tensor, P: Dict[str, torch.Tensor], mlp: dict) -> torch.Tensor:
    r = mlp["router"]
    s = torch.softmax(h @ P["router"].T, dim=-1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids = choose(s[t], P["correction"], r)
        w = s[t, ids]
        w = w / (w.sum() + 1e-20) * r["scale"]
        for e, we in zip(ids, w):
            row = h[t:t + 1]
            out[t] += we * (row if e >= r["experts"] else clamped_expert(row, P, f"e{e}.", mlp["expert"]["limit"]))[0]
    if mlp.get("shared"):
        out = out + clamped_expert(h, P, "shared.", mlp["shared"]["limit"])
    return out


def forward(cfg: dict, W: Dict[str, torch.Tensor], tokens, return_layers: bool = False):
    """Logits [T, vocab] of one whole sequence (and the residual stream after every layer)."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    norm = lambda x, name: layer_norm(x, W[name], W[name + ".b"], eps)
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    streams, v_first = [], None
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h, mix = norm(x, p + "norm1"), part(W, p + "mix.")
        if L["type"] == "parallel":
            y = two_mixers(h, mix, m, eps)
        elif L["type"] == "attention":
            y, v = attention(h, mix, m, v_first if m.get("v_mix") else None)
            if m.get("v_mix") and v_first is None:
                v_first = v
        else:
            raise ValueError(L["type"])
        x = x + mult * norm(y, p + "norm1b")
        if L.get("mlp"):
            y = expert_mixture(norm(x, p + "norm2"), part(W, p + "mlp."), L["mlp"])
            x = x + mult * norm(y, p + "norm2b")
        streams.append(x)
    logits = norm(x, "final.norm") @ W["head"].T * cfg["logit_scale"]
    cap = cfg.get("logit_softcap")
    if cap:
        logits = cap * torch.tanh(logits / cap)
    return (logits, torch.stack(streams)) if return_layers else logits
