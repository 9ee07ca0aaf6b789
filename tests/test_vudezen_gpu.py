"""Vudezen on the GPU against the plain implementation (tests/plain_vudezen.py): every mechanism's part alone through
the cache manager (requests of unequal lengths side by side, whole, in portions down to two tokens and token by token,
on pages and state slots that held other requests before), single keys made to stand out at every edge of the window and
against the sink, the recurrence's memory over hundreds of steps, the experts' choice, then whole models under every way
of cutting the work, long decoding, captured steps, and greedy generation through the engine's entry point."""
import math

import numpy as np
import pytest
import torch

import plain_vudezen as plain
import tiny_vudezen as tv
import traces
from test_simivik_gpu import (DEV, F64, Harness, _bind, _close, _compare, _dt, _i32, _junk_first, _replay, _rounded, _rt,
                              _runner, _schedules, _win_pages)

pytestmark = pytest.mark.gpu


# ============================================================================= layer norm

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("W,T", [(64, 5), (100, 5), (1000, 5), (2048, 5), (9000, 5), (1032, 300), (2048, 301), (9000, 299), (320, 300)])
def test_layer_norm_with_what_is_added_before_it(W, T, dtype):
    """A delta as it is, one that passes a norm of its own (with a bias of its own added first), and none; the stream
    is brought up to date unless rows are picked; a large mean leaves the variance alone."""
    from atom_b200.parts import registry
    from atom_b200.parts.linear import NormedDelta
    from atom_b200.parts.spec import PartSpec

    rt, dt, m = _rt(dtype), _dt(dtype), 0.37
    g = torch.Generator().manual_seed(W)
    norms, held = [], []
    for eps in (1e-5, 3e-4):
        n = registry.build("norm", PartSpec("layernorm", {"size": W, "eps": eps}))
        held.append(_bind(n, {"weight": torch.rand(W, generator=g) + 0.5, "bias": torch.randn(W, generator=g)}, rt))
        norms.append(n)
    res = torch.randn(T, W, generator=g) * 0.5 + 40.0
    delta = _rounded(torch.randn(T, W, generator=g) * 2 + 3, dtype)
    db = torch.randn(W, generator=g).to(torch.float32 if dtype == "float32" else torch.bfloat16)
    ln = lambda x, i: plain.layer_norm(x, held[i]["weight"], held[i]["bias"], norms[i].eps)
    for kind in ("none", "as it is", "normed", "normed with a bias"):
        d, add = None, 0.0
        if kind == "as it is":
            d, add = delta.to(dt).to(DEV), m * delta
        elif kind.startswith("normed"):
            b = db if kind.endswith("bias") else None
            d = NormedDelta(delta.to(dt).to(DEV), norms[1], torch.empty(T, W, dtype=dt, device=DEV), None if b is None else b.to(DEV))
            add = m * ln(delta + (0.0 if b is None else b.double()), 1)
            _close(d.run().clone(), ln(delta + (0.0 if b is None else b.double()), 1), dtype, kind + " alone", f32=2e-6, bf16=8e-3)
        want_r = res.double() + add
        rd = res.to(DEV).contiguous()
        out = norms[0].add_norm(rd, d, "t", delta_scale=m)
        _close(rd, want_r, "float32", f"{kind}: stream", f32=1e-6)
        _close(out, ln(want_r, 0), dtype, kind, f32=2e-5, bf16=8e-3)
        rd = res.to(DEV).contiguous()
        out = norms[0].add_norm(rd, d, "t2", _i32([3, 0]), 2, delta_scale=m)
        assert torch.equal(rd.cpu(), res)
        _close(out, ln(want_r[[3, 0]], 0), dtype, f"{kind}: picked rows", f32=2e-5, bf16=8e-3)


def test_a_normed_delta_of_another_kind_and_scaled_root_mean_square():
    """An RMS norm after a sub-block in front of a layer norm (two kernels), and the fused pair of RMS norms with a
    factor on what is added."""
    from atom_b200.parts import registry
    from atom_b200.parts.linear import NormedDelta
    from atom_b200.parts.spec import PartSpec

    W, T = 96, 4
    rt = _rt("float32")
    g = torch.Generator().manual_seed(1)
    rms = registry.build("norm", PartSpec("rmsnorm", {"size": W, "eps": 1e-5}))
    ln = registry.build("norm", PartSpec("layernorm", {"size": W, "eps": 1e-5}))
    hr = _bind(rms, {"weight": torch.rand(W, generator=g) + 0.5}, rt)
    hl = _bind(ln, {"weight": torch.rand(W, generator=g) + 0.5, "bias": torch.randn(W, generator=g)}, rt)
    x, res = torch.randn(T, W, generator=g), torch.randn(T, W, generator=g)
    normed = x.double() / torch.sqrt((x.double() ** 2).mean(-1, keepdim=True) + 1e-5) * hr["weight"]
    want = res.double() + 0.3 * normed
    for norm, f in ((ln, lambda r: plain.layer_norm(r, hl["weight"], hl["bias"], 1e-5)),
                    (rms, lambda r: r / torch.sqrt((r * r).mean(-1, keepdim=True) + 1e-5) * hr["weight"])):
        rd = res.to(DEV).contiguous()
        out = norm.add_norm(rd, NormedDelta(x.to(DEV), rms, torch.empty(T, W, device=DEV)), "t", delta_scale=0.3)
        _close(rd, want, "float32", "stream", f32=1e-6)
        _close(out, f(want), "float32", "norm", f32=1e-5)


# ============================================================================= attention with a sink

ATT_CASES = [  # H, G, dk, dv, rot (base, dims), yarn, window, value_mix, page, lens
    (4, 2, 16, 24, (10000.0, 8), None, 24, None, 16, (70, 9, 41)),
    (2, 1, 24, 16, None, None, None, None, 8, (50, 3, 27)),
    (3, 3, 8, 40, (77.0, 4), None, 7, None, 8, (40, 17, 2)),
    (5, 5, 20, 12, (1000.0, 12), (4.0, 40, 8.0, 1.0), 1, "mixed", 16, (33, 5, 20)),
    (6, 1, 12, 28, (300.0, 6), None, 33, "first", 16, (90, 48, 7)),
    (8, 2, 64, 32, (100000.0, 64), (8.0, 128, 32.0, 1.0), None, "mixed", 32, (300, 40, 131)),
    (4, 4, 32, 128, (10000.0, 32), None, 64, None, 16, (150, 70, 4)),
    (8, 4, 128, 128, (1000000.0, 128), (16.0, 64, 16.0, 2.0), 50, "first", 16, (140, 60, 10)),
    (6, 2, 80, 48, (10000.0, 40), None, 17, "mixed", 8, (64, 65, 63)),
    (3, 1, 7, 5, (50.0, 6), (2.0, 32, 4.0, 1.0), None, "mixed", 8, (30, 2, 11)),
    (12, 3, 48, 16, (300.0, 16), None, 129, "mixed", 16, (270, 20, 5)),
]


class _WithFirstValues:
    """A mixer that gets v_first from a matrix of the rows themselves, in place of an earlier layer."""

    def __init__(self, part, w, dt):
        self.part, self.w, self.dt = part, w.to(DEV), dt

    def cache_need(self):
        return self.part.cache_need()

    def forward(self, x, step, cache, writes_cache):
        from atom_b200.parts.sink_attention import FIRST_VALUES
        step.carried[FIRST_VALUES] = (x.float() @ self.w.T.float()).to(self.dt).contiguous()
        y = self.part.forward(x, step, cache, writes_cache)
        return y


def _attention_part(case, dtype, width=72, out_bias=True):
    from atom_b200.parts import registry
    from atom_b200.parts.spec import PartSpec

    H, G, dk, dv, rot, yarn, window, mix, page, lens = case
    m = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": 1.7 / dk ** 0.5}
    position = None
    if rot is not None:
        scaling = dict(zip(("factor", "original", "fast", "slow"), yarn)) if yarn else None
        m["rot"] = {"base": rot[0], "dims": rot[1], "scaling": scaling}
        position = PartSpec("rope_yarn", {"rotary_dim": rot[1], "theta": rot[0], "scaling": scaling, "neighbours": True})
    if window is not None:
        m["mask"] = {"size": window}
    part = registry.build("mixer", PartSpec("sink_attention", dict(
        hidden_size=width, num_heads=H, num_kv_heads=G, key_dim=dk, value_dim=dv, scale=m["scale"], position=position,
        window=window, qkv_bias=True, out_bias=out_bias, value_mix=mix)))
    g = torch.Generator().manual_seed(H * dk + dv)
    sizes = {"q": H * dk, "k": G * dk, "v": G * dv, "g": H}
    mats = {n: torch.randn(r, width, generator=g) * (2.2 if n in "qk" else 1.2) / width ** 0.5 for n, r in sizes.items()}
    names, where, w = part.layout(part.segments())
    rows = {"qkv": torch.cat([mats["q"], mats["k"], mats["v"]]), "gate": mats["g"]}
    stacked = torch.cat([rows[n] for n in names])
    t = {"in.weight": torch.cat([stacked, torch.zeros(w - stacked.shape[0], width)]),
         "o.weight": torch.randn(width, H * dv, generator=g) / (H * dv) ** 0.5,
         "qkv.bias": torch.randn(sum(sizes[n] for n in "qkv"), generator=g) * 0.5, "sink": torch.rand(H, generator=g) * 3}
    if out_bias:
        t["o.bias"] = torch.randn(width, generator=g) * 0.3
    if mix:
        t["vmix"] = torch.tensor([0.625])
    held = _bind(part, t, _rt(dtype))
    P = {"sink": held["sink"], "o": held["o.weight"]}
    if out_bias:
        P["o.b"] = held["o.bias"]
    a, n = where["qkv"]
    at = 0
    for s in "qkv":
        P[s], P[s + ".b"] = held["in.weight"][a + at:a + at + sizes[s]], held["qkv.bias"][at:at + sizes[s]]
        at += sizes[s]
    P["g"] = held["in.weight"][where["gate"][0]:where["gate"][0] + H]
    P["vmix"] = 0.625
    return part, m, P, width


@pytest.mark.parametrize("dtype", ["float32", "bfloat16", "bfloat16-plain"])
@pytest.mark.parametrize("case", ATT_CASES)
def test_sink_attention_part_under_every_cut(case, dtype, monkeypatch):
    """(bfloat16 runs the tensor-core kernel where it takes the sizes; "bfloat16-plain" the plain kernel there too.)"""
    from atom_b200 import native
    if dtype.endswith("-plain"):
        if not native.window_attention_tc_supports(case[2], case[3], torch.bfloat16):
            pytest.skip("these sizes run the plain kernel anyway")
        monkeypatch.setattr(native, "WINDOW_TC", False)
        dtype = "bfloat16"
    part, m, P, W = _attention_part(case, dtype)
    G, dv, mix, page, lens = case[1], case[3], case[7], case[8], dict(zip("abc", case[9]))
    g = torch.Generator().manual_seed(sum(case[9]))
    x = {r: _rounded(torch.randn(n, W, generator=g), dtype) for r, n in lens.items()}
    first = (torch.randn(G * dv, W, generator=g) / W ** 0.5).float()
    v_first = {r: None for r in lens}
    if mix == "mixed":
        v_first = {r: (x[r].float() @ first.T).to(_dt(dtype)).double().view(-1, G, dv) for r in lens}
    want = {r: plain.attention(x[r], P, m, v_first[r])[0] for r in lens}
    driven = _WithFirstValues(part, first, _dt(dtype)) if mix == "mixed" else part
    for what, sched in _schedules(lens):
        h = Harness(driven, dtype, page=page, pages=3 * (max(lens.values()) // page + 3))
        _junk_first(h, W)
        got = h.run(x, sched)
        for r in lens:
            _close(got[r], want[r], dtype, f"{what}, request {r}", f32=3e-5, bf16=3e-2)
        assert all(gr.pool.num_used == 0 for gr in h.manager.groups) and h.manager.state_slots.num_free == 4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_layers_values_are_carried_to_the_layers_that_blend(dtype):
    """The layer that blends first leaves its values (with their bias, before rotation of anything) for the step's later
    layers; a bias left to the arrangement is left out of the output."""
    case = (4, 2, 16, 24, (100.0, 8), None, None, "first", 8, (11,))
    part, m, P, W = _attention_part(case, dtype)
    g = torch.Generator().manual_seed(5)
    x = _rounded(torch.randn(11, W, generator=g), dtype)
    want, v = plain.attention(x, P, m)
    seen = {}

    class Spy(_WithFirstValues):
        def forward(self, rows, step, cache, writes_cache):
            y = self.part.forward(rows, step, cache, writes_cache)
            seen["v"] = next(iter(step.carried.values())).clone()
            return y
    part.leave_bias = True
    assert part.late_bias is not None
    got = Harness(Spy(part, torch.zeros(1), _dt(dtype)), dtype).run({"a": x}, [{"a": 11}])["a"]
    _close(seen["v"], v.reshape(11, -1), dtype, "values", f32=1e-5, bf16=1e-2)
    _close(got + P["o.b"], want, dtype, "output", f32=3e-5, bf16=3e-2)


def _kernels(dk, dv, dtype):
    from atom_b200 import native
    return ["plain", "tc1", "tc3", "tc7"] if native.window_attention_tc_supports(dk, dv, _dt(dtype)) else ["plain"]


def _run_attention(q, k, v, scale, window, sink, gate, out_scale, dtype, page, cuts, kernel):
    """One request's keys and values in scrambled pages, the queries in portions ``cuts``; the output is a part of wider
    rows (the rest must stay as it was)."""
    from atom_b200 import native

    T, H, dk = q.shape
    G, dv = k.shape[1], v.shape[2]
    dt = _dt(dtype)
    table, kp, vp = _win_pages(T, G, page, dk, dv, dtype, seed=T)
    out = torch.zeros(T, H * dv, dtype=dt, device=DEV)
    sk = sink.float().to(DEV).contiguous() if sink is not None else None
    at = 0
    for n in cuts:
        n = min(n, T - at)
        if n <= 0:
            continue
        j = torch.arange(at, at + n, device=DEV)
        pg = table[0].long()[j // page]
        kp[pg, :, j % page] = k[at:at + n].to(dt).to(DEV)
        vp[pg, :, j % page] = v[at:at + n].to(dt).to(DEV)
        wide = torch.full((n, H * dv + 16), 9.0, dtype=dt, device=DEV)
        o = wide[:, 8:8 + H * dv]
        gt = None
        if gate is not None:
            gt = torch.zeros(n, H + 5, dtype=dt, device=DEV)[:, 3:3 + H]
            gt.copy_(gate[at:at + n].to(dt))
        qd = q[at:at + n].reshape(n, H * dk).to(dt).to(DEV).contiguous()
        kw = dict(sink=sk, gate=gt, out_scale=out_scale)
        if kernel.startswith("tc"):
            ns = int(kernel[2:])
            scratch = torch.full((native.attention_mixed_scratch_elems(n, H, dv, ns),), float("nan"), dtype=torch.float32,
                                 device=DEV) if ns > 1 else None
            native.window_attention_tc(o, qd, kp, vp, table, _i32(range(at, at + n)), _i32([0] * n), _i32([0, n]), 1, H, G,
                                       dk, dv, scale, 0.0, window, 0, ns, scratch, heads_rows=(n == 1 and at % 2 == 0), **kw)
        else:
            native.window_attention(o, qd, kp, vp, table, _i32(range(at, at + n)), _i32([0] * n), H, G, dk, dv, scale,
                                    0.0, window, 0, **kw)
        assert bool((wide[:, :8] == 9).all()) and bool((wide[:, 8 + H * dv:] == 9).all())
        out[at:at + n] = o
        at += n
    assert at == T
    return out.double().cpu().view(T, H, dv)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window", [1, 2, 16, 17, 64, 65, 300, 0])
def test_single_keys_at_the_windows_edge_with_a_sink_and_a_gate(window, dtype):
    """A key row that carries a mark only it has and a score far above all others: seen at distance window - 1, not at
    distance window (window 0: from everywhere after it), in a prompt, across portions that end at every place around the
    edge and a page's border, and decoded one by one.  A sink as large as the mark's score takes half of its weight, and a
    head whose sink is far above it nearly all."""
    H, G, dk, dv, page, T = 4, 2, 32, 16, 16, 420
    needle = 95
    g = torch.Generator().manual_seed(window)
    k = torch.randn(T, G, dk, generator=g) * 0.1
    v = torch.randn(T, G, dv, generator=g) * 0.1
    q = torch.randn(T, H, dk, generator=g) * 0.1
    v[:, :, 0] = 0.0
    k[:, :, 0] = 0.0
    q[:, :, 0] = 3.0
    v[needle, :, 0], k[needle, :, 0] = 1.0, 4.0                # a score of 12 against a few tenths
    q, k, v = _rounded(q, dtype), _rounded(k, dtype), _rounded(v, dtype)
    sink = torch.tensor([-50.0, 12.0, 3.0, 40.0], dtype=F64)
    gate = _rounded(torch.randn(T, H, generator=g), dtype)
    ungated = plain.sink_attention(q, k, v, 1.0, sink, window or None)
    want = ungated * torch.sigmoid(gate)[:, :, None] * 1.25
    sees = lambda i: i >= needle and (not window or i - needle < window)
    for i in range(T):
        assert (float(ungated[i, 0, 0]) > 0.9 and 0.4 < float(ungated[i, 1, 0]) < 0.6 and float(ungated[i, 3, 0]) < 1e-6) == sees(i)
    edge = needle + (window or 200)
    cut_sets = [[T], [edge - 1, 1, 1, 1, T], [edge, T], [edge + 1, T], [needle, 2, window or 9, 2, T]]
    if 0 < window <= 65:
        cut_sets.append([needle + 1] + [1] * (T - needle - 1))
    for cuts in cut_sets:
        for kernel in _kernels(dk, dv, dtype):
            if kernel in ("tc3", "tc7") and len(cuts) > 20:
                continue
            got = _run_attention(q, k, v, 1.0, window, sink, gate, 1.25, dtype, page, cuts, kernel)
            what = f"{kernel}, window {window}, cuts {cuts[:4]}"
            marks = got[:, 0, 0] / (torch.sigmoid(gate[:, 0]) * 1.25)
            for i in range(T):
                assert (float(marks[i]) > 0.8) if sees(i) else (float(marks[i]) == 0), f"{what}: key {needle} from {i}"
            _close(got, want, dtype, what, f32=2e-5, bf16=1e-2)


@pytest.mark.parametrize("H,G,dk,dv,window,page,T", [(8, 2, 64, 32, 0, 32, 333), (12, 3, 96, 32, 100, 16, 300),
                                                      (4, 1, 128, 128, 70, 16, 270), (3, 3, 48, 16, 65, 8, 200)])
def test_tensor_core_attention_with_a_sink_against_plain(H, G, dk, dv, window, page, T):
    g = torch.Generator().manual_seed(T + dk)
    q, k = (_rounded(torch.randn(T, n, dk, generator=g), "bfloat16") for n in (H, G))
    v = _rounded(torch.randn(T, G, dv, generator=g), "bfloat16")
    sink = torch.rand(H, generator=g).double() * 6 - 2
    gate = _rounded(torch.randn(T, H, generator=g) * 2, "bfloat16")
    scale = 3.0 / dk ** 0.5
    want = plain.sink_attention(q, k, v, scale, sink.float().double(), window or None) * torch.sigmoid(gate)[:, :, None]
    kernels = _kernels(dk, dv, "bfloat16")
    assert "tc1" in kernels
    for kernel in kernels:
        for cuts in ([T], [T - 9] + [1] * 9, [13, 64, 5, 2, 129, 2, 70, 3, 17] * 8):
            got = _run_attention(q, k, v, scale, window, sink, gate, 1.0, "bfloat16", page, cuts, kernel)
            _close(got, want, "bfloat16", f"{kernel}, cuts {cuts[:3]}", bf16=1e-2)


# ============================================================================= the state-space recurrence

SSM_CASES = [  # heads, vdim, state, groups, taps, norm_groups, lens
    (6, 8, 12, 3, 3, 2, (70, 9, 41)),
    (4, 16, 16, 4, 1, 1, (37, 5, 18)),
    (5, 9, 3, 5, 10, 5, (50, 2, 31)),
    (1, 21, 33, 1, 5, 3, (33, 64, 65)),
    (4, 64, 64, 2, 4, 4, (300, 40, 131)),
    (8, 64, 128, 2, 4, 2, (150, 3, 70)),
    (2, 32, 256, 1, 2, 1, (130, 65, 7)),
    (3, 40, 20, 1, 8, 3, (2500, 7, 200)),
    (4, 48, 32, 2, 4, 2, (200, 129, 16)),
]


def _ssm_part(case, dtype, width=72):
    from atom_b200.parts import registry
    from atom_b200.parts.spec import PartSpec

    H, P_, N, G, taps, parts, lens = case
    eps = 2e-5
    m = {"heads": H, "vdim": P_, "state": N, "groups": G, "conv": taps, "norm_groups": parts}
    part = registry.build("mixer", PartSpec("state_space", dict(
        hidden_size=width, num_heads=H, value_dim=P_, state_dim=N, groups=G, taps=taps, norm_groups=parts, norm_eps=eps)))
    g = torch.Generator().manual_seed(H * P_ + N)
    I, C = H * P_, H * P_ + 2 * G * N
    w = torch.randn(I + C + H, width, generator=g) * 1.5 / width ** 0.5
    cw = torch.randn(C, taps, generator=g) * (0.5 / taps ** 0.5)
    cw[:, -1] += 0.8
    uni = lambda n, lo, hi: torch.rand(n, generator=g) * (hi - lo) + lo
    spec = part.params()["in.weight"]
    t = {"in.weight": torch.cat([w, torch.zeros(spec.pad, width)]), "o.weight": torch.randn(width, I, generator=g) / I ** 0.5,
         "conv.weight": cw, "conv.bias": torch.randn(C, generator=g) * 0.3, "dt_bias": uni(H, -3.0, 0.5),
         "A_log": uni(H, -4.0, 1.0), "D": uni(H, -1.0, 1.5), "norm": uni(I, 0.7, 1.3)}
    held = _bind(part, t, _rt(dtype))
    P = {"in": held["in.weight"][:I + C + H], "o": held["o.weight"], "conv": held["conv.weight"], "conv.b": held["conv.bias"],
         "dt_bias": held["dt_bias"], "A_log": held["A_log"], "D": held["D"], "norm": held["norm"]}
    return part, m, P, eps, width


@pytest.mark.parametrize("dtype", ["float32", "bfloat16", "bfloat16-plain"])
@pytest.mark.parametrize("case", SSM_CASES)
def test_state_space_part_under_every_cut(case, dtype, monkeypatch):
    """The state and the convolution's rows go from step to step in the request's slot, whatever the cut (also steps
    with fewer rows than taps); steps of many rows take the forms that work on runs of rows side by side (bfloat16 on the
    tensor cores where the sizes allow, "bfloat16-plain" on plain FMAs there too)."""
    from atom_b200 import native
    if dtype.endswith("-plain"):
        if case[1] % 8 or case[2] % 8:
            pytest.skip("these sizes run the plain kernel anyway")
        monkeypatch.setattr(native, "SSM_TC", False)
        dtype = "bfloat16"
    part, m, P, eps, W = _ssm_part(case, dtype)
    lens = dict(zip("abc", case[6]))
    g = torch.Generator().manual_seed(sum(case[6]))
    x = {r: _rounded(torch.randn(n, W, generator=g), dtype) for r, n in lens.items()}
    want = {r: plain.mamba2(x[r], P, m, eps) for r in lens}
    for what, sched in _schedules(lens):
        if what == "pairs" and max(lens.values()) > 1000:
            continue
        h = Harness(part, dtype)
        _junk_first(h, W)
        got = h.run(x, sched)
        for r in lens:
            _close(got[r], want[r], dtype, f"{what}, request {r}", f32=5e-5, bf16=4e-2)
        assert h.manager.state_slots.num_free == 4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16", "bfloat16-plain"])
@pytest.mark.parametrize("H,G,N,P_,T", [(4, 2, 64, 64, 700), (6, 3, 12, 8, 200), (2, 1, 128, 64, 333), (2, 2, 32, 48, 130),
                                        (3, 1, 24, 136, 190), (2, 1, 256, 32, 128), (4, 4, 8, 72, 257)])
def test_scan_in_runs_equals_the_scan_token_by_token(H, G, N, P_, T, dtype, monkeypatch):
    """The same rows in one step (runs side by side) and one by one, and against the plain recurrence, with decays from
    almost none to a factor of e^-8 a token; several requests side by side, each beginning with a state that is not zero."""
    from atom_b200 import native

    if dtype.endswith("-plain"):
        monkeypatch.setattr(native, "SSM_TC", False)
        dtype = "bfloat16"
    dt_ = _dt(dtype)
    g = torch.Generator().manual_seed(T)
    lens = [T, 1, 65]
    n = sum(lens)
    u = _rounded(torch.randn(n, H * P_ + 2 * G * N, generator=g), dtype)
    dt = torch.rand(n, H, generator=g) * 0.8 + 0.05
    A = torch.exp(torch.linspace(-6.0, 2.3, H))
    la = -A[None] * dt
    D = _rounded(torch.randn(H, generator=g), "float32").float()
    S0 = torch.randn(4, H, N, P_, generator=g)
    cu = [0, lens[0], lens[0] + lens[1], n]

    def run(state, rows, cu_q, slots):
        R = rows[1] - rows[0]
        o = torch.empty(R, H * P_, dtype=torch.float32, device=DEV)
        nb, na = native.ssm_scratch_elems(R, len(slots), H, N, P_, native.ssm_run(R, N, P_, dt_)[0])
        sb = torch.full((max(nb, 1),), float("nan"), device=DEV)
        sa = torch.full((max(na, 1),), float("nan"), device=DEV)
        sl = slice(rows[0], rows[1])
        native.ssm_scan(o, u[sl].to(dt_).to(DEV).contiguous(), dt[sl].to(DEV).contiguous(), la[sl].to(DEV).contiguous(), D.to(DEV),
                        state, sb if nb else None, sa if na else None, _i32(cu_q), _i32(slots), len(slots), H, G, N, P_, True)
        return o.double().cpu()
    st = S0.to(DEV).contiguous()
    got = run(st, (0, n), cu, [2, 0, 3])
    assert torch.equal(st[1].cpu(), S0[1])                                   # another request's slot is left alone
    per = H // G
    for slot, a, b in ((2, cu[0], cu[1]), (0, cu[1], cu[2]), (3, cu[2], cu[3])):
        x, B, C = torch.split(u[a:b], [H * P_, G * N, G * N], dim=1)
        x = x.view(-1, H, P_)
        B, C = (t.reshape(-1, G, N).repeat_interleave(per, dim=1) for t in (B, C))
        S, y = S0[slot].double(), []
        for t in range(b - a):
            S = torch.exp(la[a + t].double())[:, None, None] * S + dt[a + t].double()[:, None, None] * B[t][:, :, None] * x[t][:, None, :]
            y.append(torch.einsum("hnp,hn->hp", S, C[t]) + D.double()[:, None] * x[t])
        y = torch.stack(y).reshape(b - a, -1)
        # (32-bit throughout: the sums' own size is what roundings scale with, not the activations' type)
        _close(got[a:b], y, "float32", f"slot {slot}", f32=1e-5)
        _close(st[slot], S, "float32", f"state {slot}", f32=1e-5)
    one = S0.to(DEV).contiguous()
    for t in range(80):
        o = run(one, (t, t + 1), [0, 1], [2])
        _close(o, got[t:t + 1], "float32", f"token {t}", scale=float(got.abs().max()), f32=1e-5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_state_after_six_hundred_single_steps(dtype):
    """One input at step 2, then nothing but the same C for 600 steps of one token: the output falls as exp(-A dt n), in
    32-bit whatever the activations' type (a state kept in 16 bits would stop falling, or fall to zero at once)."""
    from atom_b200 import native

    H, P_, N, n = 3, 8, 16, 600
    dt_ = _dt(dtype)
    A = torch.tensor([0.001, 0.03, 1e-6])
    state = torch.full((2, H, N, P_), 7.0, dtype=torch.float32, device=DEV)
    state[1].zero_()
    outs = []
    for t in range(n):
        u = torch.zeros(1, H * P_ + 2 * N, dtype=dt_, device=DEV)
        u[:, H * P_ + N:] = 1.5                                                  # C
        if t == 2:
            u[:, :H * P_ + N] = 2.0                                              # x and B
        o = torch.empty(1, H * P_, dtype=torch.float32, device=DEV)
        d = torch.full((1, H), 0.5, device=DEV)
        native.ssm_scan(o, u, d, -A[None].to(DEV) * d, torch.zeros(H, device=DEV), state, None, None, _i32([0, 1]), _i32([1]),
                        1, H, 1, N, P_, True)
        outs.append(o[0].double().cpu().view(H, P_))
    assert float(outs[1].abs().max()) == 0
    want = torch.exp(-A.double() * 0.5 * (n - 3)) * 0.5 * 4.0 * 1.5 * N
    _close(outs[-1][:, 0], want, "float32", "after 600 steps", f32=1e-4)
    assert bool((state[0] == 7.0).all())


def test_step_sizes_have_no_clamp():
    from atom_b200 import native

    raw = torch.tensor([[-200.0, -20.0, -1.0, 0.0, 3.0, 25.0, 300.0]], device=DEV)
    H, z = raw.shape[1], lambda *n: torch.zeros(*n, device=DEV)
    b, a_log = torch.full((H,), 0.25, device=DEV), torch.linspace(-3, 2, H, device=DEV)
    for taps in (1, 4, 9):
        dt, la = torch.full((1, H), -1.0, device=DEV), torch.full((1, H), 1.0, device=DEV)
        rows = torch.cat([z(1, 5), raw], dim=1)
        native.ssm_conv(z(1, 5), rows[:, :5], z(5, taps), z(5), z(2, taps - 1, 5) if taps > 1 else None, dt, la, rows[:, 5:], b,
                        a_log, _i32([0]), _i32([0, 1]), _i32([1]), 1)
        _check_steps(dt, la, raw, a_log)


def _check_steps(dt, la, raw, a_log):
    v = raw.double().cpu() + 0.25
    want = torch.log1p(torch.exp(-v.abs())) + v.clamp(min=0)
    assert torch.allclose(dt.double().cpu(), want, rtol=1e-6, atol=1e-40)
    assert torch.allclose(la.double().cpu(), -torch.exp(a_log.double().cpu()) * want, rtol=1e-6, atol=1e-40)


# ============================================================================= two mixers, their outputs added

PAIR_CASES = [  # attention case, state-space case (without lens), scales, lens
    (ATT_CASES[0], SSM_CASES[0], (1.3, 0.7), (70, 9, 41)),
    (ATT_CASES[3][:7] + (None,) + ATT_CASES[3][8:], SSM_CASES[3], (0.6, 1.2), (33, 64, 3)),
    (ATT_CASES[6], SSM_CASES[4], (1.0, -0.5), (140, 70, 5)),
    (ATT_CASES[4][:7] + (None,) + ATT_CASES[4][8:], SSM_CASES[2], (2.0, 1.0), (50, 2, 31)),
]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", PAIR_CASES)
def test_summed_mixers_under_every_cut(case, dtype):
    """One stacked projection, one output matrix over both members' rows; each member's rows carry its factor."""
    from atom_b200.parts import registry
    from atom_b200.parts.spec import PartSpec

    att, ssm, (ls, rs), lengths = case
    W = 72
    left, ml, Pl, _ = _attention_part(att, dtype, W, out_bias=False)
    right, mr, Pr, eps, _ = _ssm_part(ssm, dtype, W)
    specs = {}
    for n, p in (("left", left), ("right", right)):
        specs[n] = PartSpec(p.kind, _args_of(p, att if n == "left" else ssm, ml if n == "left" else mr, W, eps))
    part = registry.build("mixer", PartSpec("summed_mixers", {"hidden_size": W, "members": specs, "scales": {"left": ls, "right": rs}}))
    names, where, width = part.layout(part.segments())
    own = {"left.qkv": torch.cat([Pl["q"], Pl["k"], Pl["v"]]), "left.gate": Pl["g"], "right.in": Pr["in"]}
    stacked = torch.cat([own[n] for n in names])
    t = {"in.weight": torch.cat([stacked, torch.zeros(width - stacked.shape[0], W, dtype=F64)]),
         "o.weight": torch.cat([Pl["o"], Pr["o"]], dim=1), "left.qkv.bias": torch.cat([Pl["q.b"], Pl["k.b"], Pl["v.b"]]),
         "left.sink": Pl["sink"], "right.conv.weight": Pr["conv"], "right.conv.bias": Pr["conv.b"]}
    t.update({f"right.{n}": Pr[n] for n in ("dt_bias", "A_log", "D", "norm")})
    _bind(part, t, _rt(dtype))
    P = {**{f"left.{k}": v for k, v in Pl.items() if k != "vmix"}, **{f"right.{k}": v for k, v in Pr.items()}}
    lens = dict(zip("abc", lengths))
    g = torch.Generator().manual_seed(sum(lengths))
    x = {r: _rounded(torch.randn(n, W, generator=g), dtype) for r, n in lens.items()}
    want = {r: plain.two_mixers(x[r], P, {"left": ml, "left_scale": ls, "right": mr, "right_scale": rs}, eps) for r in lens}
    for what, sched in _schedules(lens):
        h = Harness(part, dtype, page=att[8], pages=3 * (max(lens.values()) // att[8] + 3))
        _junk_first(h, W)
        got = h.run(x, sched)
        for r in lens:
            _close(got[r], want[r], dtype, f"{what}, request {r}", f32=5e-5, bf16=4e-2)
        assert all(gr.pool.num_used == 0 for gr in h.manager.groups) and h.manager.state_slots.num_free == 4


def _args_of(part, case, m, W, eps):
    from atom_b200.parts.spec import PartSpec
    if part.kind == "state_space":
        return dict(hidden_size=W, num_heads=m["heads"], value_dim=m["vdim"], state_dim=m["state"], groups=m["groups"],
                    taps=m["conv"], norm_groups=m["norm_groups"], norm_eps=eps)
    position = None
    if m.get("rot"):
        position = PartSpec("rope_yarn", {"rotary_dim": m["rot"]["dims"], "theta": m["rot"]["base"],
                                          "scaling": m["rot"]["scaling"], "neighbours": True})
    return dict(hidden_size=W, num_heads=m["heads"], num_kv_heads=m["kv_heads"], key_dim=m["dim"], value_dim=m["vdim"],
                scale=m["scale"], position=position, window=m["mask"]["size"] if m.get("mask") else None, qkv_bias=True)


# ============================================================================= experts

EXPERT_CASES = [  # width, experts, identity, top, groups, ff, limit, shared (ff, limit), factor, T
    (64, 6, 2, 2, (4, 2), 24, 1.1, (40, 0.8), 1.7, 45),
    (96, 5, 0, 3, None, 40, 2.0, (24, 1.5), 1.0, 33),
    (100, 3, 0, 3, None, 28, 0.7, (36, 2.5), 0.4, 7),
    (72, 2, 4, 2, (2, 1), 12, 1.4, None, 1.0, 130),
    (72, 1, 0, 1, None, 16, 1.0, (8, 0.5), 1.0, 1),
    (128, 16, 4, 4, (5, 3), 64, 1.5, None, 2.0, 300),
    (192, 40, 24, 8, (64, 33), 72, 0.9, (64, 1.0), 1.5, 70),
    (256, 8, 4, 2, (3, 1), 128, 1.2, (256, 1.5), 2.0, 700),
    (136, 6, 3, 4, (3, 2), 18, 3.0, None, 3.0, 16),
]


def _expert_part(case, dtype):
    from atom_b200.parts import registry
    from atom_b200.parts.spec import PartSpec

    W, E, ident, top, groups, ff, limit, shared, factor, T = case
    part = registry.build("ffn", PartSpec("routed_experts", dict(
        hidden_size=W, num_experts=E, top=top, intermediate_size=ff, shared_size=shared[0] if shared else None,
        score="softmax", renormalize=True, weight_on="output", correction=True, groups=groups, identity=ident, factor=factor,
        sum_eps=1e-20, limit=limit, shared_limit=shared[1] if shared else None)))
    g = torch.Generator().manual_seed(W + E)
    mat = lambda o, i, gain=1.0: torch.randn(o, i, generator=g) * gain / i ** 0.5
    t = {"router.weight": mat(E + ident, W, 2.0), "correction": torch.randn(E + ident, generator=g) * 0.2 - 0.5,
         "gate_up.weight": torch.cat([mat(ff, W, 1.5) for _ in range(2 * E)]),
         "down.weight": torch.cat([mat(W, ff, 1.5) for _ in range(E)])}
    if shared:
        t["shared.gate_up.weight"] = torch.cat([mat(shared[0], W, 1.5), mat(shared[0], W, 1.5)])
        t["shared.down.weight"] = mat(W, shared[0], 1.5)
    held = _bind(part, t, _rt(dtype))
    P = {"router": held["router.weight"], "correction": held["correction"]}
    for e in range(E):
        P[f"e{e}.gate"] = held["gate_up.weight"][2 * e * ff:(2 * e + 1) * ff]
        P[f"e{e}.up"] = held["gate_up.weight"][(2 * e + 1) * ff:(2 * e + 2) * ff]
        P[f"e{e}.down"] = held["down.weight"][e * W:(e + 1) * W]
    router = {"experts": E, "top": top, "scale": factor}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    mlp = {"router": router, "expert": {"limit": limit}}
    if shared:
        S = shared[0]
        P["shared.gate"], P["shared.up"] = held["shared.gate_up.weight"][:S], held["shared.gate_up.weight"][S:]
        P["shared.down"] = held["shared.down.weight"]
        mlp["shared"] = {"limit": shared[1]}
    x = _rounded(torch.randn(T, W, generator=g), dtype)
    if T > 40:
        x[5:25] = x[5]                        # twenty rows with the same choice: an expert with many rows
    return part, P, mlp, x


@pytest.mark.parametrize("dtype", ["float32", "bfloat16", "bfloat16-plain"])
@pytest.mark.parametrize("case", EXPERT_CASES)
def test_clamped_experts_with_groups_and_identities(case, dtype, monkeypatch):
    """All choice scores are negative here (a barred expert must count as less than any of them).  Rows whose choice
    hangs on less than the projection's rounding are left out of the bfloat16 comparison."""
    from types import SimpleNamespace

    from atom_b200 import native
    if dtype.endswith("-plain"):
        monkeypatch.setattr(native, "MOE_TC", False)
        dtype = "bfloat16"
    part, P, mlp, x = _expert_part(case, dtype)
    T = x.shape[0]
    want = plain.expert_mixture(x, P, mlp)
    clear = torch.ones(T, dtype=torch.bool)
    if dtype == "bfloat16":
        s = torch.softmax(x @ P["router"].T, -1)
        for t in range(T):
            for sign in (-1, 1):
                noise = sign * 1e-3 * torch.cos(torch.arange(s.shape[1], dtype=F64) * 2.1 + t)
                clear[t] &= set(plain.choose(s[t] + noise, P["correction"], mlp["router"])) == set(plain.choose(s[t], P["correction"], mlp["router"]))
        assert clear.double().mean() > 0.8
    step = SimpleNamespace(seq_of_token=_i32([0] * T), num_tokens=T, num_seqs=1)
    for _ in range(2):                        # twice: what the first call leaves in the workspace does not leak
        got = part.forward(x.to(_dt(dtype)).to(DEV), step)
        _close(got.cpu()[clear], want[clear], dtype, "experts", f32=3e-5, bf16=3e-2)


@pytest.mark.parametrize("counts,N,K", [
    ([300, 0, 1, 128, 129, 0, 255, 256, 257], 192, 136), ([0, 0, 700], 520, 64), ([64] * 40, 64, 320), ([1], 8, 8),
    ([513, 2, 127, 90], 1032, 200), ([5, 4, 0, 3, 2, 1], 256, 512), ([0, 0], 128, 128), ([2600, 1500], 768, 256)])
def test_grouped_products_on_tcgen05(counts, N, K):
    """Every expert's rows against its own matrix: experts without rows, rows that end anywhere in a tile, sizes that end
    anywhere in a tile; rows behind the last expert's are left alone, gathered rows are the right ones."""
    from atom_b200 import native

    g = torch.Generator().manual_seed(sum(counts) + N)
    E, n = len(counts), sum(counts)
    R = n + 37
    off = torch.tensor([0] + counts).cumsum(0).to(torch.int32)
    src = torch.randn(50, K, generator=g).to(torch.bfloat16)
    tok = torch.randint(0, 50, (R,), generator=g).to(torch.int32)
    wts = torch.rand(R, generator=g)
    for weighted in (False, True):
        x = torch.full((R, K), float("nan"), dtype=torch.bfloat16, device=DEV)
        native.moe_gather(x, src.to(DEV), off.to(DEV), E, tok.to(DEV), wts.to(DEV) if weighted else None)
        rows = src[tok.long()][:n]
        rows = (rows.float() * wts[:n, None]).to(torch.bfloat16) if weighted else rows
        assert torch.equal(x.cpu()[:n], rows) and bool(x[n:].isnan().all())
    for gated, act in ((False, "silu"), (True, "silu"), (True, "clamped")):
        w = (torch.randn(E, (2 if gated else 1) * N, K, generator=g) * 2 / K ** 0.5).to(torch.bfloat16)
        out = torch.full((R, N), 7.0, dtype=torch.bfloat16, device=DEV)
        native.gemm_pairs_grouped(x, w.to(DEV), out, off.to(DEV), gated, act, 1.25)
        torch.cuda.synchronize()
        native.check_error_flags()
        assert bool((out[n:] == 7).all())
        for e in range(E):
            r = rows[off[e]:off[e + 1]].double()
            we = w[e].double()
            if not gated:
                want = r @ we.T
            elif act == "silu":
                want = torch.nn.functional.silu(r @ we[:N].T) * (r @ we[N:].T)
            else:
                want = plain.clamped_expert(r, {"gate": we[:N], "up": we[N:], "down": torch.eye(N, dtype=F64)}, "", 1.25)
            if counts[e]:
                _close(out[off[e]:off[e + 1]], want, "bfloat16", f"expert {e}, {act if gated else 'plain'}", bf16=1.5e-2)


def test_router_choice_kernel_with_groups_corrections_and_identities():
    from atom_b200 import native

    g = torch.Generator().manual_seed(5)
    for n, ident, top, groups, shift, T in ((8, 2, 2, (4, 2), -2.0, 60), (64, 8, 8, (8, 3), 0.0, 300), (200, 100, 32, (10, 2), -5.0, 17),
                                            (96, 0, 4, (48, 40), 1.0, 33), (12, 3, 3, (1, 1), 0.0, 40), (1024, 24, 6, (128, 100), -1.0, 9)):
        logits = torch.randn(T, n + 3, generator=g) * 2
        corr = torch.randn(n, generator=g) * 0.3 + shift
        ids = torch.empty(T, top, dtype=torch.int32, device=DEV)
        wts = torch.empty(T, top, dtype=torch.float32, device=DEV)
        counts = torch.zeros(1024, dtype=torch.int32, device=DEV)
        native.moe_route(logits.to(DEV), n, top, "softmax", True, _i32([0] * T), ids, wts, counts, ident, 1e-20, 2.5,
                         corr.to(DEV), *groups)
        s = torch.softmax(logits[:, :n].double(), -1)
        got = ids.cpu().long()
        for t in range(T):
            ref = plain.choose(s[t], corr.double(), {"top": top, "groups": {"count": groups[0], "keep": groups[1]}})
            c = s[t] + corr.double()
            # the same experts, or ones whose choice score is the same to 32-bit rounding
            assert sorted(got[t].tolist()) == sorted(ref) or torch.allclose(c[got[t]].sort().values, c[ref].sort().values, atol=3e-7)
        w = torch.gather(s, 1, got)
        _close(wts, w / w.sum(-1, keepdim=True) * 2.5, "float32", "weights", f32=2e-6)
        rows = got[got < n - ident]
        assert torch.equal(counts[:n].cpu().long(), torch.bincount(rows, minlength=n))


@pytest.mark.parametrize("T,I,K", [(3, 64, 128), (16, 136, 192), (40, 72, 64), (40, 9, 40), (700, 1024, 256)])
def test_clamped_gate_in_every_gated_product(T, I, K):
    """Few rows (the streaming product's epilogue), some (library product and activation kernel), many (the tcgen05
    product's epilogue); the limit bites on a good part of the numbers."""
    from atom_b200.parts.linear import gated_linear

    g = torch.Generator().manual_seed(T)
    for dtype in ("bfloat16", "float32"):
        dt = _dt(dtype)
        x = _rounded(torch.randn(T, K, generator=g), dtype)
        w = _rounded(torch.randn(2 * I, K, generator=g) * 2 / K ** 0.5, dtype)
        out = torch.empty(T, I, dtype=dt, device=DEV)
        got = gated_linear(x.to(dt).to(DEV), w.to(dt).to(DEV), out, lambda m, n: torch.empty(m, n, dtype=dt, device=DEV),
                           "clamped", 1.25)
        P = {"gate": w[:I], "up": w[I:], "down": torch.eye(I, dtype=F64)}
        _close(got, plain.clamped_expert(x, P, "", 1.25), dtype, f"{T} x {I}", f32=1e-5, bf16=1.5e-2)


def test_logits_are_scaled_then_capped():
    from atom_b200.parts import registry
    from atom_b200.parts.spec import PartSpec

    g = torch.Generator().manual_seed(2)
    for cap in (0.0, 4.0):
        head = registry.build("head", PartSpec("lm_head", {"vocab_size": 70, "hidden_size": 64, "tied": False, "scale": 3.0, "softcap": cap}))
        w = _bind(head, {"weight": torch.randn(70, 64, generator=g)}, _rt("float32"))["weight"]
        x = torch.randn(5, 64, generator=g)
        want = x.double() @ w.T * 3.0
        assert float(want.abs().max()) > 40
        got = head.forward(x.to(DEV))
        _close(got, cap * torch.tanh(want / cap) if cap else want, "float32", f"cap {cap}", f32=1e-5)


# ============================================================================= whole models

LENGTHS = {"A": [1, 2, 9, 41, 100, 70], "B": [3, 17, 64, 131, 30], "C": [5, 33, 90, 48, 70], "D": [4, 70, 150, 33],
           "R": [3, 40, 75]}


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    out = {}
    for name, cfg in tv.CONFIGS.items():
        d = str(tmp_path_factory.mktemp(f"vudezen_{name}"))
        tv.write_model(cfg, d, tv.SEEDS[name], free_choice=name == "R")
        out[name] = d
    return out


_plain_memo = {}


def _plain_logits(model_dir, seqs):
    if model_dir not in _plain_memo:
        _plain_memo[model_dir] = tv.read_model(model_dir) + ({},)
    cfg, w, memo = _plain_memo[model_dir]
    out = {}
    for rid, toks in seqs.items():
        key = tuple(toks)
        if key not in memo:
            memo[key] = plain.forward(cfg, w, list(toks)).numpy()
        out[rid] = memo[key]
    return out


def _seqs(name):
    ps = tv.prompts(tv.CONFIGS[name], LENGTHS[name], seed=len(name) + ord(name))
    return {f"r{i}": p for i, p in enumerate(ps)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_layer_by_layer_against_plain(dirs, name, dtype):
    """The residual stream after every layer of a short prompt (what the next norm reads)."""
    from atom_b200.engine.batch import StepEntry
    from atom_b200.parts.linear import NormedDelta
    cfg, w = tv.read_model(dirs[name])
    p = tv.prompts(tv.CONFIGS[name], [45], seed=2)[0]
    want = plain.forward(cfg, w, p, return_layers=True)[1]
    runner = _runner(dirs[name], dtype, 64, tv.PAGE[name])
    seen = []
    for b in runner.model.blocks:
        def run(residual, delta, step, cache, wc, delta_scale=None, _o=b.run, _b=b):
            out = _o(residual, delta, step, cache, wc, delta_scale=delta_scale)
            assert isinstance(out, NormedDelta)
            x, x_bias = out.x.clone(), out.x_bias
            seen.append(residual.double() + _b.delta_scale * NormedDelta(x, out.norm, torch.empty_like(x), x_bias).run().double())
            return out
        b.run = run
    runner.step([StepEntry("a", p, [0])])
    runner.check_status()
    assert len(seen) == len(want) == len(cfg["layers"])
    for i, (g, r) in enumerate(zip(seen, want)):
        _close(g, r, dtype, f"after layer {i}", f32=3e-5, bf16=3e-2)


@pytest.mark.parametrize("name,dtype", [(n, d) for n in tv.CONFIGS for d in ("float32", "bfloat16") if n != "R" or d == "float32"])
def test_every_cut_matches_plain(dirs, name, dtype):
    """Whole; the last 48 tokens one by one (every window of these models but one passes over decoded tokens); portions of
    changing size down to two tokens; pairs of tokens throughout; up to four live requests with portions beside single
    tokens in a pool so small that pages and state slots are used again."""
    seqs = _seqs(name)
    ref = _plain_logits(dirs[name], seqs)
    mixed, peak = traces.mixed(seqs, max_live=4, budget_tokens=320)
    assert peak <= 320 and (name == "R" or 320 < sum(-(-len(t) // 64) * 64 for t in seqs.values()))
    runner = _runner(dirs[name], dtype, 320, tv.PAGE[name], max_num_seqs=4)
    for what, steps in (("whole", traces.whole(seqs)), ("tail", traces.tail_by_token(seqs, 48)),
                        ("ragged", traces.ragged(seqs)), ("pairs", traces.ragged(seqs, sizes=(2,))), ("mixed", mixed)):
        if what == "pairs":
            steps = [s for s in steps if s["entries"][0]["id"] in ("r1", "r2")]       # (two short requests are enough)
            sub = {r: ref[r] for r in ("r1", "r2")}
            _compare(traces.collect(steps, _replay(runner, steps)), sub, dtype, f"{name}/{what}")
            continue
        _compare(traces.collect(steps, _replay(runner, steps)), ref, dtype, f"{name}/{what}")
        assert all(g.pool.num_used == 0 for g in runner.cache.groups) and runner.cache.state_slots.num_free == 4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_request_freed_half_way_and_fed_again(dirs, name, dtype):
    """What preemption by recomputation does: pages and the state slot go back, another request takes them, and the
    victim starts over on whatever slot is free, with a state and a convolution tail of zeros."""
    seqs = _seqs(name)
    ref = _plain_logits(dirs[name], seqs)
    ids = list(seqs)
    steps, peak = traces.mixed_refeed(seqs, [ids[-1], ids[-2]], max_live=3, budget_tokens=384)
    runner = _runner(dirs[name], dtype, peak, tv.PAGE[name], max_num_seqs=3)
    rows = traces.collect_rows(steps, _replay(runner, steps))
    scale = max(float(np.abs(r).max()) for r in ref.values())
    tol = {"float32": 2e-4, "bfloat16": 8e-2}[dtype] * max(1.0, scale)
    for rid, got in rows.items():
        assert {p for p, _ in got} == set(range(len(seqs[rid])))
        errs = [float(np.abs(row.astype(np.float64) - ref[rid][p]).max()) for p, row in got]
        assert max(errs) <= tol, f"{name}/{dtype}: {rid}: worst {max(errs):.3e} > {tol:.3e}"
    assert all(g.pool.num_used == 0 for g in runner.cache.groups) and runner.cache.state_slots.num_free == 3


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batch_of_unequal_requests_equals_each_alone(dirs, dtype):
    """The same rows, computed alone and beside three other requests of other lengths, differ by rounding at most."""
    name = "D"
    ps = tv.prompts(tv.CONFIGS[name], [50, 3, 27, 64], seed=99)
    runner = _runner(dirs[name], dtype, 1024, tv.PAGE[name])
    from atom_b200.engine.batch import StepEntry
    alone = []
    for i, p in enumerate(ps):
        alone.append(runner.step([StepEntry(("a", i), p, list(range(len(p))))]).float().cpu().numpy())
        runner.finish(("a", i))
    both = runner.step([StepEntry(("b", i), p, list(range(len(p)))) for i, p in enumerate(ps)]).float().cpu().numpy()
    at = 0
    for i, p in enumerate(ps):
        part = both[at:at + len(p)]
        at += len(p)
        scale = float(np.abs(alone[i]).max())
        assert np.abs(part - alone[i]).max() <= (1e-4 if dtype == "float32" else 4e-2) * scale
    runner.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding_token_by_token(dirs, name, dtype):
    """300 tokens decoded one by one after a prompt of three: pages fill, follow one another and, where there is a window,
    are given back; the recurrent state and the convolution's tail are read and written 300 times."""
    p = tv.prompts(tv.CONFIGS[name], [303], seed=4)[0]
    seqs = {"long": p}
    ref = _plain_logits(dirs[name], seqs)
    steps = traces.tail_by_token(seqs, 300)
    runner = _runner(dirs[name], dtype, 304, tv.PAGE[name])
    _compare(traces.collect(steps, _replay(runner, steps)), ref, dtype, "long decoding")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_captured_steps_match_plain(dirs, dtype):
    """Decode steps and small mixed steps replayed from CUDA graphs, with padding rows and padding requests."""
    name = "A"
    seqs = _seqs(name)
    ref = _plain_logits(dirs[name], seqs)
    runner = _runner(dirs[name], dtype, 1024, tv.PAGE[name], max_num_seqs=8, enforce_eager=False,
                     cudagraph_capture_sizes=[1, 2, 4], max_model_len=256)
    for what, steps in (("tail", traces.tail_by_token(seqs, 32)), ("mixed", traces.mixed(seqs, max_live=3, tail=40)[0]),
                        ("ragged", traces.ragged(seqs))):
        _compare(traces.collect(steps, _replay(runner, steps)), ref, dtype, f"graphs/{what}")
    assert runner.graph_replays > 50
    assert all(g.pool.num_used == 0 for g in runner.cache.groups)


def _plain_greedy(cfg, w, prompt, n_new):
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(plain.forward(cfg, w, ids)[-1].argmax()))
    return ids[len(prompt):]


@pytest.mark.parametrize("name,chunk", [("A", 8), ("C", 13)])
def test_greedy_generation_through_the_engine_fp32(dirs, name, chunk):
    from atom_b200 import LLMEngine, SamplingParams
    cfg, w = tv.read_model(dirs[name])
    prompts = tv.prompts(tv.CONFIGS[name], [1, 7, 16, 33], seed=21)
    eng = LLMEngine(dirs[name], dtype="float32", kv_cache_block_size=tv.PAGE[name], num_kvcache_blocks=64,
                    enforce_eager=(name == "C"), max_num_batched_tokens=chunk + 4, long_prefill_token_threshold=chunk,
                    max_num_seqs=4)
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=10, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert o["num_tokens_output"] == 10
        assert o["token_ids"] == _plain_greedy(cfg, w, p, 10)
    assert all(g.pool.num_used == 0 for g in eng.runner.cache.groups)


def test_greedy_generation_bf16_with_preemption(dirs):
    """A pool so small that requests are preempted and computed again; every token stays within rounding of the
    plain implementation's best."""
    from atom_b200 import LLMEngine, SamplingParams
    name = "B"
    cfg, w = tv.read_model(dirs[name])
    prompts = tv.prompts(tv.CONFIGS[name], [3, 5, 12, 29], seed=5)
    eng = LLMEngine(dirs[name], dtype="bfloat16", kv_cache_block_size=8, num_kvcache_blocks=14, max_num_batched_tokens=24,
                    max_num_seqs=4, enforce_eager=True)
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=40, ignore_eos=True))
    assert eng.stats()["preemptions"] > 0
    for p, o in zip(prompts, outs):
        full = list(p) + o["token_ids"]
        logits = plain.forward(cfg, w, full[:-1]).numpy()
        for i, tok in enumerate(o["token_ids"]):
            row = logits[len(p) - 1 + i]
            assert row[tok] >= row.max() - 0.03 * np.abs(logits).max(), f"token {i}: logit {row[tok]:.3f} against {row.max():.3f}"
    eng.runner.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_program_on_a_vudezen_folder(dirs, tmp_path, dtype):
    """bin/trace_run as a user runs it (a child process, steps on standard input, one file of logits per step): the
    model class is chosen by config.json; four state slots and a pool smaller than the requests' sum."""
    import json
    import os
    import subprocess
    import sys

    name = "A"
    seqs = _seqs(name)
    steps, peak = traces.mixed(seqs, max_live=4, budget_tokens=320)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / f"out_{dtype}"
    text = "".join(json.dumps(s) + "\n" for s in steps)
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", dirs[name], "--dtype", dtype,
                        "--out", str(out), "--max-tokens", str(peak)], input=text, capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [int(l.split()[1]) for l in p.stdout.splitlines() if l.startswith("done ")] == [s["step"] for s in steps]
    V = tv.CONFIGS[name]["vocab"]
    outputs = {}
    for s in steps:
        n = sum(len(e["want"]) for e in s["entries"])
        if n:
            a = np.fromfile(out / f"{s['step']}.f32", dtype="<f4")
            assert a.size == n * V
            outputs[s["step"]] = a.reshape(n, V)
    _compare(traces.collect(steps, outputs), _plain_logits(dirs[name], seqs), dtype, f"trace_run/{dtype}")
