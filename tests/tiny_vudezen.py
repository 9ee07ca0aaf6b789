"""Tiny Vudezen configurations that differ in every size, constant and in the order of layers, and a writer of model
folders with seeded random weights (bfloat16 storage) whose scales make the attention sharp, the sinks and the biases
large, the recurrence's memory long, and the routers' choices clear, so that a wrong key, a window that is one token off,
a lost state, a missing sink or a wrong expert shows.

A: both kinds of layers in turn; groups of experts with identity experts; one layer without a feed-forward; YaRN.
B: attention without rotation and without blended values first; no groups, no identity or no shared expert; a window
   wider than any prompt; one tap; as many groups as heads; plain rotary frequencies.
C: sizes that are multiples of 4 but not of 8 or odd, an odd vocabulary, a window of one token, more taps than the
   convolution's fast kernel takes, every expert chosen, a cap off, three layers that blend values.
D: sizes of the order of real models' heads, a window of 100.
R: as A, with corrections that change most choices (only for 32-bit: a choice may hang on little).
"""
from __future__ import annotations

import copy
import json
import os
from typing import Dict, List, Optional

import numpy as np
import torch


def _att(heads, kv_heads, dim, vdim, scale, rot=None, yarn=None, window=None, v_mix=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if yarn is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    if window is not None:
        m["mask"] = {"size": window}
    if v_mix is not None:
        m["v_mix"] = v_mix
    return m


def _ssm(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def _pair(left, ls, right, rs):
    return {"left": left, "left_scale": ls, "right": right, "right_scale": rs}


def _moe(experts, top, ff, limit, identity=None, groups=None, shared=None, scale=1.0):
    r = {"experts": experts, "top": top, "scale": scale}
    if identity is not None:
        r["identity"] = identity
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    m = {"kind": "moe", "router": r, "expert": {"ff": ff, "limit": limit}}
    if shared is not None:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def _layer(mixer, mlp=None):
    return {"type": "parallel" if "left" in mixer else "attention", "mixer": mixer, "mlp": mlp}


def _cfg(vocab, width, eps, m, scale, cap, layers):
    c = {"architecture": "Vudezen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": m,
         "logit_scale": scale, "layers": layers}
    if cap is not None:
        c["logit_softcap"] = cap
    return c


_LEFT_A = _att(4, 2, 16, 24, 0.3, rot=(10000.0, 8), window=24)
_MOE_A = _moe(6, 2, 24, 1.1, identity=2, groups=(4, 2), shared=(40, 0.8), scale=1.7)
_FULL_A = _att(3, 1, 24, 8, 0.25, rot=(500.0, 24), yarn=(4.0, 40, 8.0, 1.0), v_mix=True)

CONFIGS: Dict[str, dict] = {
    "A": _cfg(211, 64, 1e-5, 0.6, 1.5, 12.0,
              [_layer(_pair(_LEFT_A, 1.3, _ssm(6, 8, 12, 3, 3, 2), 0.7), _MOE_A), _layer(_FULL_A, _MOE_A),
               _layer(_pair(_LEFT_A, 0.9, _ssm(2, 24, 20, 1, 4, 3), 1.1)), _layer(_FULL_A, _MOE_A)]),
    "B": _cfg(300, 96, 1e-6, 0.9, 0.8, 30.0,
              [_layer(_att(2, 1, 24, 16, 0.2, v_mix=False), _moe(5, 3, 40, 2.0, shared=(24, 1.5))),
               _layer(_pair(_att(3, 3, 8, 40, 0.35, rot=(77.0, 4), window=1000), 0.5, _ssm(4, 16, 16, 4, 1, 1), 1.5),
                      _moe(4, 1, 32, 0.9, identity=1)),
               _layer(_att(6, 2, 8, 8, 0.4, rot=(10000.0, 8), v_mix=True), _moe(7, 2, 20, 1.2, groups=(7, 3))),
               _layer(_pair(_att(4, 4, 16, 16, 0.3, rot=(1000.0, 16), window=7), 1.2, _ssm(3, 32, 8, 3, 2, 2), 0.8), None)]),
    "C": _cfg(257, 100, 3e-5, 0.45, 2.2, None,
              [_layer(_att(5, 5, 20, 12, 0.22, rot=(1000.0, 12), v_mix=True), _moe(3, 3, 28, 0.7, shared=(36, 2.5), scale=0.4)),
               _layer(_pair(_att(6, 1, 12, 28, 0.3, rot=(300.0, 6), window=1), 0.7, _ssm(5, 9, 3, 5, 10, 5), 1.2), None),
               _layer(_att(5, 5, 10, 12, 0.3, rot=(5000.0, 10), yarn=(16.0, 64, 4.0, 2.0), v_mix=True),
                      _moe(2, 2, 12, 1.4, identity=4, groups=(2, 1))),
               _layer(_att(10, 5, 14, 12, 0.25, v_mix=True), _moe(6, 4, 18, 3.0, identity=3, groups=(3, 2), scale=3.0)),
               _layer(_pair(_att(2, 2, 4, 7, 0.5, window=33), 1.0, _ssm(1, 21, 33, 1, 5, 3), 1.0), _moe(1, 1, 16, 1.0, shared=(8, 0.5)))]),
    "D": _cfg(512, 256, 1e-5, 0.7, 1.2, 20.0,
              [_layer(_att(4, 2, 128, 64, 0.09, rot=(100000.0, 64), yarn=(8.0, 128, 32.0, 1.0), v_mix=True),
                      _moe(8, 2, 128, 1.2, identity=4, groups=(3, 1), shared=(256, 1.5), scale=2.0)),
               _layer(_pair(_att(8, 2, 64, 32, 0.125, rot=(100000.0, 32), window=100), 1.1, _ssm(4, 64, 64, 2, 4, 4), 0.9),
                      _moe(16, 4, 64, 1.5, groups=(4, 2), scale=1.5)),
               _layer(_att(6, 2, 96, 64, 0.1, rot=(10000.0, 96), v_mix=True), None)]),
}
CONFIGS["R"] = copy.deepcopy(CONFIGS["A"])
SEEDS = {"A": 7, "B": 8, "C": 4, "D": 13, "R": 21}
PAGE = {"A": 16, "B": 8, "C": 16, "D": 32, "R": 16}


def _outputs(mlp) -> int:
    return mlp["router"]["experts"] + mlp["router"].get("identity", 0)


def random_tensors(cfg: dict, seed: int, overrides: Optional[Dict[str, torch.Tensor]] = None,
                   free_choice: bool = False) -> Dict[str, torch.Tensor]:
    """free_choice: corrections of the size of the scores' differences (else one expert that is always and one that is
    never chosen, and the tokens' own levels between them)."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    R = max([_outputs(L["mlp"]) for L in cfg["layers"] if L["mlp"]] or [0])
    t: Dict[str, torch.Tensor] = {}

    def mat(out, inp, gain=1.0):
        return torch.randn(out, inp, generator=g) * (gain / inp ** 0.5)

    def uni(n, lo, hi):
        return torch.rand(n, generator=g) * (hi - lo) + lo

    def norm(name, gain=1.0, quiet=False):
        w, b = uni(W, 0.7, 1.3) * gain, uni(W, -0.3, 0.3) * gain
        if quiet and R:          # (the stream's last numbers, which the routers read, stay almost as the embedding has them)
            w[W - R:] *= 0.04
            b[W - R:] = 0.0
        t[name], t[name + ".b"] = w, b

    emb = torch.randn(V, W, generator=g)
    levels = torch.arange(R, dtype=torch.float32) - (R - 1) / 2
    for v in range(V if R else 0):       # every token ranks the experts in an order of its own, a level apart
        emb[v, W - R:] = levels[torch.randperm(R, generator=g)] * (3.0 / R)
    t["embed"], t["head"] = emb, mat(V, W, 2.0)
    norm("final.norm")

    def attention(p, m, out_bias):
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        sharp = (2.5 / (m["scale"] * d ** 0.5)) ** 0.5             # scores of a few units: a sharp softmax
        for n, rows, gain in (("q", H * d, sharp), ("k", G * d, sharp), ("v", G * dv, 1.0)):
            t[p + n] = mat(rows, W, gain)
            t[p + n + ".b"] = torch.randn(rows, generator=g) * 0.4
        t[p + "sink"], t[p + "g"] = uni(H, 0.0, 4.0), mat(H, W, 1.5)
        t[p + "o"] = mat(W, H * dv)
        if out_bias:
            t[p + "o.b"] = torch.randn(W, generator=g) * 0.3
        if m.get("v_mix"):
            t[p + "vmix"] = uni(1, 0.3, 0.7)[0]

    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        norm(p + "norm1")
        norm(p + "norm1b", quiet=True)
        if L["type"] == "attention":
            attention(p + "mix.", m, True)
        else:
            attention(p + "mix.left.", m["left"], False)
            r, rp = m["right"], p + "mix.right."
            inner, C = r["heads"] * r["vdim"], r["heads"] * r["vdim"] + 2 * r["groups"] * r["state"]
            t[rp + "in"] = mat(inner + C + r["heads"], W, 1.5)
            cw = torch.randn(C, r["conv"], generator=g) * (0.5 / r["conv"] ** 0.5)
            cw[:, -1] += 0.8
            t[rp + "conv"], t[rp + "conv.b"] = cw, torch.randn(C, generator=g) * 0.3
            t[rp + "dt_bias"], t[rp + "A_log"] = uni(r["heads"], -2.5, 0.5), uni(r["heads"], -4.0, 0.5)
            t[rp + "D"], t[rp + "norm"] = uni(r["heads"], -1.0, 1.5), uni(inner, 0.7, 1.3)
            t[rp + "o"] = mat(W, inner)
        mlp = L["mlp"]
        if mlp is None:
            continue
        E, n, ff = mlp["router"]["experts"], _outputs(mlp), mlp["expert"]["ff"]
        norm(p + "norm2")
        t[p + "norm2"][W - R:], t[p + "norm2.b"][W - R:] = 1.0, 0.0
        norm(p + "norm2b", quiet=True)
        router = mat(n, W, 0.03)
        router[:, W - R:] = 0.0
        router[:, W - R:W - R + n] += torch.eye(n) * (R / 3.0)          # reads the token's level for this expert
        t[p + "mlp.router"] = router
        c = torch.zeros(n)
        if free_choice:
            c = torch.randn(n, generator=g) * 0.3
        elif n > mlp["router"]["top"] + 1:
            order = torch.randperm(n, generator=g)
            c[order[0]], c[order[1]] = 1.0, -1.0
        t[p + "mlp.correction"] = c
        for e in range(E):
            t[p + f"mlp.e{e}.gate"], t[p + f"mlp.e{e}.up"] = mat(ff, W, 1.5), mat(ff, W, 1.5)
            t[p + f"mlp.e{e}.down"] = mat(W, ff)
        if mlp.get("shared"):
            S = mlp["shared"]["ff"]
            t[p + "mlp.shared.gate"], t[p + "mlp.shared.up"] = mat(S, W, 1.5), mat(S, W, 1.5)
            t[p + "mlp.shared.down"] = mat(W, S)
    if overrides:
        for k, v in overrides.items():
            assert t[k].shape == v.shape, k
            t[k] = v
    return {k: v.to(torch.bfloat16).contiguous() for k, v in t.items()}


def write_model(cfg: dict, model_dir: str, seed: int, overrides: Optional[Dict[str, torch.Tensor]] = None,
                free_choice: bool = False) -> None:
    from safetensors.torch import save_file

    os.makedirs(model_dir, exist_ok=True)
    with open(os.path.join(model_dir, "config.json"), "w") as f:
        json.dump(cfg, f, indent=1)
    save_file(random_tensors(cfg, seed, overrides, free_choice), os.path.join(model_dir, "model.safetensors"),
              metadata={"format": "pt"})


def read_model(model_dir: str):
    """(config dict, {name: float64 tensor}) for the plain implementation."""
    from safetensors.torch import load_file

    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, {k: v.double() for k, v in load_file(os.path.join(model_dir, "model.safetensors")).items()}


def prompts(cfg: dict, lengths: List[int], seed: int) -> List[List[int]]:
    rng = np.random.default_rng(seed)
    return [rng.integers(0, cfg["vocab"], size=n).tolist() for n in lengths]
