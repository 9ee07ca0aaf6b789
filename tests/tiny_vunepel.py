"""Tiny Vunepel configurations that differ in every size, constant and in the order of layers, and a writer of model
folders with seeded random weights (bfloat16 storage) whose scales make both attention maps sharp, the recurrence's memory
long and its writes strong, and the routers' choices clear, so that a wrong key, a chunk that is one token off, a lost
state, a missing convolution row or a wrong expert shows.

A: both kinds of mixers in turn, shared keys read within chunks of another size, dense and expert feed-forwards.
B: attention first, over everything and without rotation; shared keys read by two layers; one tap; as many key heads as
   heads; a layer without a feed-forward; experts without a shared one.
C: sizes that are multiples of 4 but not of 8 or odd, an odd vocabulary, chunks of one token, more taps than the fast
   convolution takes, every expert chosen, ranks of 1 and 5.
D: sizes of the order of real models' heads, chunks of 100, many heads per key head.
E: no attention at all.
"""
from __future__ import annotations

import json
import os
from typing import Dict, List

import numpy as np
import torch


def _att(heads, kv_heads, dim, vdim, scale, diff, rot=None, chunk=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def _delta(heads, kv_heads, dim, vdim, conv, ranks):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": ranks[0],
            "gate_rank": ranks[1]}


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _moe(experts, top, ff, limit, shared=None, scale=1.0):
    m = {"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale}, "expert": {"ff": ff, "limit": limit}}
    if shared is not None:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def _layer(mixer, mlp=None):
    return {"type": "channel_delta" if "conv" in mixer else "attention", "mixer": mixer, "mlp": mlp}


def _cfg(vocab, width, eps, layers):
    return {"architecture": "Vunepel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


_ROT_A = (10000.0, 8)
CONFIGS: Dict[str, dict] = {
    "A": _cfg(211, 64, 1e-5, [
        _layer(_delta(4, 2, 16, 24, 4, (8, 16)), _dense(72, 1.2)),
        _layer(_att(4, 2, 16, 24, 0.3, 0.35, _ROT_A, 24), _moe(6, 2, 24, 1.1, (40, 0.8), 1.7)),
        _layer(_delta(2, 1, 24, 8, 2, (16, 8)), _moe(5, 3, 32, 0.9, (24, 2.0), 0.8)),
        _layer(_att(6, 2, 16, 24, 0.25, 0.6, _ROT_A, 40, kv_from=1), _dense(40, 0.7))]),
    "B": _cfg(300, 96, 1e-6, [
        _layer(_att(2, 1, 24, 16, 0.2, 0.2), _moe(5, 3, 40, 2.0)),
        _layer(_delta(3, 3, 32, 16, 1, (24, 40)), None),
        _layer(_att(4, 1, 24, 16, 0.4, 0.8, chunk=7, kv_from=0), _moe(4, 1, 32, 0.9, scale=2.0)),
        _layer(_att(6, 3, 8, 40, 0.35, 0.5, (77.0, 4), 16), _dense(56, 1.5)),
        _layer(_att(1, 1, 24, 16, 0.3, 0.1, kv_from=0), None)]),
    "C": _cfg(257, 100, 3e-5, [
        _layer(_delta(6, 3, 10, 7, 10, (5, 1)), _dense(30, 0.6)),
        _layer(_att(5, 5, 20, 12, 0.22, 0.45, (1000.0, 12), 1), _moe(3, 3, 28, 0.7, (36, 2.5), 0.4)),
        _layer(_delta(5, 1, 13, 33, 3, (1, 11)), None),
        _layer(_att(6, 2, 6, 9, 0.4, 0.3, (300.0, 6), 33), _moe(7, 4, 18, 3.0, (8, 0.5), 3.0)),
        _layer(_att(4, 2, 6, 9, 0.5, 0.7, (300.0, 6), 50, kv_from=3), None)]),
    "D": _cfg(512, 256, 1e-5, [
        _layer(_delta(4, 2, 128, 64, 4, (64, 32)), _dense(512, 1.5)),
        _layer(_att(8, 1, 64, 128, 0.125, 0.4, (100000.0, 64), 100), _moe(8, 2, 128, 1.2, (256, 1.5), 2.0)),
        _layer(_delta(2, 2, 64, 128, 4, (32, 64)), _moe(16, 4, 64, 1.5, (64, 1.0), 1.5)),
        _layer(_att(4, 1, 64, 128, 0.1, 0.65, (100000.0, 64), 100, kv_from=1), _dense(256, 1.0))]),
    "E": _cfg(150, 48, 1e-5, [
        _layer(_delta(2, 2, 16, 16, 3, (8, 8)), _dense(48, 1.0)),
        _layer(_delta(4, 1, 8, 16, 5, (8, 4)), _moe(4, 2, 16, 1.0, (16, 1.0), 1.3))]),
}
SEEDS = {"A": 7, "B": 8, "C": 4, "D": 13, "E": 6}
PAGE = {"A": 16, "B": 8, "C": 16, "D": 32, "E": 16}


def random_tensors(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    R = max([L["mlp"]["router"]["experts"] for L in cfg["layers"] if L["mlp"] and L["mlp"]["kind"] == "moe"] or [0])
    t: Dict[str, torch.Tensor] = {}

    def mat(out, inp, gain=1.0):
        return torch.randn(out, inp, generator=g) * (gain / inp ** 0.5)

    def uni(n, lo, hi):
        return torch.rand(n, generator=g) * (hi - lo) + lo

    def norm(name):
        w, b = uni(W, 0.8, 1.6), uni(W, -0.3, 0.3)
        w[W - R:], b[W - R:] = 1.0, 0.0
        t[name], t[name + ".b"], t[name + ".alpha"] = w, b, uni(1, 0.4, 0.9)[0]

    def quiet(m):           # (the stream's last numbers, which the routers read, stay almost as the embedding has them)
        m[W - R:] *= 0.03
        return m

    emb = torch.randn(V, W, generator=g)
    levels = torch.arange(R, dtype=torch.float32) - (R - 1) / 2
    for v in range(V if R else 0):       # every token ranks the experts in an order of its own, a level apart
        emb[v, W - R:] = levels[torch.randperm(R, generator=g)] * (3.0 / R)
    t["embed"], t["head"] = emb, mat(V, W, 2.0)
    norm("final.norm")

    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        norm(p + "norm1")
        q = p + "mix."
        if L["type"] == "attention":
            sharp = (3.0 / (m["scale"] * d ** 0.5)) ** 0.5             # scores of a few units: a sharp softmax
            t[q + "q"], t[q + "q.norm"] = mat(H * 2 * d, W), uni(d, 0.7, 1.3) * sharp
            if m.get("kv_from") is None:
                t[q + "k"], t[q + "k.norm"] = mat(G * 2 * d, W), uni(d, 0.7, 1.3) * sharp
                t[q + "v"] = mat(G * dv, W, 1.5)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                t[q + n] = torch.randn(d, generator=g) * (0.6 / d ** 0.25)
        else:
            for n, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
                t[q + n] = mat(rows, W, 1.5)
                cw = torch.randn(rows, m["conv"], generator=g) * (0.5 / m["conv"] ** 0.5)
                cw[:, -1] += 0.8
                t[q + n + ".conv"] = cw
            t[q + "b"], t[q + "A_log"], t[q + "dt_bias"] = mat(H, W, 2.0), uni(H, -4.0, 0.5), uni(H * d, -2.5, 0.5)
            t[q + "a1"], t[q + "a2"] = mat(m["decay_rank"], W), mat(H * d, m["decay_rank"])
            t[q + "g1"], t[q + "g2"] = mat(m["gate_rank"], W, 2.0), mat(H * dv, m["gate_rank"])
            t[q + "norm"] = uni(dv, 0.7, 1.3)
        t[q + "o"] = quiet(mat(W, H * dv))
        mlp, q = L["mlp"], p + "mlp."
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            ff = mlp["ff"]
            t[q + "gate"], t[q + "up"], t[q + "down"] = mat(ff, W, 1.5), mat(ff, W, 1.5), quiet(mat(W, ff))
            continue
        n, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
        router = mat(n, W, 0.03)
        router[:, W - R:] = 0.0
        router[:, W - R:W - R + n] += torch.eye(n) * (R / 3.0)          # reads the token's level for this expert
        t[q + "router"] = router
        for e in range(n):
            t[q + f"e{e}.gate"], t[q + f"e{e}.up"] = mat(ff, W, 1.5), mat(ff, W, 1.5)
            t[q + f"e{e}.down"] = quiet(mat(W, ff))
        if mlp.get("shared"):
            S = mlp["shared"]["ff"]
            t[q + "shared.gate"], t[q + "shared.up"] = mat(S, W, 1.5), mat(S, W, 1.5)
            t[q + "shared.down"], t[q + "shared.sg"] = quiet(mat(W, S)), mat(1, W, 1.5)
    return {k: v.to(torch.bfloat16).contiguous() for k, v in t.items()}


def write_model(cfg: dict, model_dir: str, seed: int) -> None:
    """(the ranks stand in the tensors' shapes alone, as in a checkpoint)"""
    from safetensors.torch import save_file

    os.makedirs(model_dir, exist_ok=True)
    bare = json.loads(json.dumps(cfg))
    for L in bare["layers"]:
        L["mixer"].pop("decay_rank", None)
        L["mixer"].pop("gate_rank", None)
    with open(os.path.join(model_dir, "config.json"), "w") as f:
        json.dump(bare, f, indent=1)
    save_file(random_tensors(cfg, seed), os.path.join(model_dir, "model.safetensors"), metadata={"format": "pt"})


def read_model(model_dir: str):
    """(config dict, {name: float64 tensor}) for the plain implementation."""
    from safetensors.torch import load_file

    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, {k: v.double() for k, v in load_file(os.path.join(model_dir, "model.safetensors")).items()}


def prompts(cfg: dict, lengths: List[int], seed: int) -> List[List[int]]:
    rng = np.random.default_rng(seed)
    return [rng.integers(0, cfg["vocab"], size=n).tolist() for n in lengths]
