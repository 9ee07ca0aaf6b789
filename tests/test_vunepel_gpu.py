"""Vunepel on the GPU against the plain implementation (tests/plain_vunepel.py): every mechanism's part alone through the
cache manager (requests of unequal lengths side by side, whole, in portions down to two tokens and token by token, on pages
and state slots that held other requests before), single keys made to stand out at every chunk's border and in either map,
the recurrence's memory over hundreds of steps, then whole models under every way of cutting the work, long decoding,
captured steps, and greedy generation through the engine's entry point."""
import numpy as np
import pytest
import torch

import plain_vunepel as plain
import tiny_vunepel as tv
import traces
from test_simivik_gpu import (DEV, F64, Harness, _bind, _close, _compare, _dt, _i32, _junk_first, _replay, _rounded, _rt,
                              _runner, _schedules, _win_pages)

pytestmark = pytest.mark.gpu


def _part(category, kind, **args):
    from atom_b200.parts import registry
    from atom_b200.parts.spec import PartSpec
    return registry.build(category, PartSpec(kind, args))


# ============================================================================= dynamic tanh

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("W,T", [(64, 5), (100, 5), (1000, 7), (2048, 300), (5001, 3), (9000, 40), (8, 1)])
def test_dynamic_tanh_with_one_or_two_outputs_added_before_it(W, T, dtype):
    from atom_b200.parts.linear import SumDelta

    rt, dt = _rt(dtype), _dt(dtype)
    g = torch.Generator().manual_seed(W)
    norm = _part("norm", "dynamic_tanh", size=W)
    held = _bind(norm, {"weight": torch.rand(W, generator=g) + 0.5, "bias": torch.randn(W, generator=g),
                        "alpha": torch.tensor([0.71])}, rt)
    f = lambda r: plain.dynamic_tanh(r, held["weight"], held["bias"], held["alpha"])
    res = torch.randn(T, W, generator=g) * 2
    a, b = (_rounded(torch.randn(T, W, generator=g), dtype) for _ in range(2))
    dev = lambda x: x.to(dt).to(DEV).contiguous()
    for what, delta, add in (("none", None, 0.0), ("one", dev(a), a), ("two", SumDelta(dev(a), dev(b)), a + b)):
        want = res.double() + add
        rd = res.to(DEV).contiguous()
        out = norm.add_norm(rd, delta, "t")
        _close(rd, want, "float32", f"{what}: stream", f32=1e-6)
        _close(out, f(want), dtype, what, f32=2e-6, bf16=5e-3)
        pick = [T - 1, 0]
        rd = res.to(DEV).contiguous()
        out = norm.add_norm(rd, delta, "t2", _i32(pick), 2)
        assert torch.equal(rd.cpu(), res)
        _close(out, f(want[pick]), dtype, f"{what}: picked rows", f32=2e-6, bf16=5e-3)
    rd = res.to(DEV).contiguous()
    SumDelta(dev(a), dev(b)).add_to(rd)
    _close(rd, res.double() + a + b, "float32", "added without a norm", f32=1e-6)


def test_two_outputs_before_a_norm_that_adds_one(tmp_path):
    """A model whose last norm (or next layer) does not add two outputs itself gets the sum in the stream."""
    import dataclasses

    from atom_b200.config import EngineConfig
    from atom_b200.config.model_config import load_model_config
    from atom_b200.engine.batch import StepEntry
    from atom_b200.engine.runner import ModelRunner
    from atom_b200.models import registry as models
    from atom_b200.parts.spec import PartSpec

    tv.write_model(tv.CONFIGS["E"], str(tmp_path), 6)
    cfg = load_model_config(str(tmp_path))
    arch = models.get_architecture("Vunepel")
    spec = arch.build_spec(cfg)
    rms = PartSpec("rmsnorm", {"size": cfg.width, "eps": 1e-5}, {"weight": ("final.norm",)})
    other = dataclasses.replace(spec, final_norm=rms, ignored_tensors=(r"final\.norm\.(b|alpha)",))
    models._ARCHITECTURES["Vunepel"] = dataclasses.replace(arch, build_spec=lambda c: other)
    try:
        runner = ModelRunner(EngineConfig(model=str(tmp_path), dtype="float32", num_kvcache_blocks=4, max_num_seqs=2, enforce_eager=True))
    finally:
        models._ARCHITECTURES["Vunepel"] = arch
    p = tv.prompts(tv.CONFIGS["E"], [20], 1)[0]
    got = runner.step([StepEntry("a", p, list(range(20)))])
    c, w = tv.read_model(str(tmp_path))
    x = plain.forward(c, w, p, return_layers=True)[1][-1]
    _close(got, plain.rms(x, 1e-5) * w["final.norm"] @ w["head"].T, "float32", "logits", f32=2e-5)


# ============================================================================= gated delta rule

DELTA_CASES = [  # heads, kv_heads, dim, vdim, taps, ranks, lens
    (4, 2, 16, 24, 4, (8, 16), (70, 9, 41)),
    (3, 3, 32, 16, 1, (24, 40), (37, 5, 18)),
    (6, 3, 10, 7, 10, (5, 1), (50, 2, 31)),
    (5, 1, 13, 33, 3, (1, 11), (33, 64, 65)),
    (4, 2, 128, 64, 4, (64, 32), (300, 40, 131)),
    (2, 2, 64, 128, 2, (32, 64), (150, 3, 70)),
    (2, 1, 256, 32, 3, (16, 16), (130, 65, 7)),
    (2, 2, 96, 40, 8, (16, 16), (700, 7, 200)),
    (4, 4, 64, 64, 4, (16, 24), (200, 129, 16)),
    (3, 1, 128, 128, 4, (16, 24), (193, 64, 63)),
    (1, 1, 1, 1, 2, (1, 1), (40, 3, 9)),
    (2, 1, 32, 144, 4, (8, 8), (200, 100, 5)),
    (2, 2, 60, 100, 3, (8, 8), (130, 3, 70)),
]
EPS = 2e-5


def _delta_part(case, dtype, width=72):
    H, G, d, dv, taps, (ra, rg), lens = case
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv}
    part = _part("mixer", "channel_delta_rule", hidden_size=width, num_heads=H, num_kv_heads=G, key_dim=d, value_dim=dv,
                 taps=taps, decay_rank=ra, gate_rank=rg, norm_eps=EPS)
    g = torch.Generator().manual_seed(H * d + dv)
    mat = lambda o, i, gain=1.0: torch.randn(o, i, generator=g) * gain / i ** 0.5
    uni = lambda n, lo, hi: torch.rand(n, generator=g) * (hi - lo) + lo
    sizes = {"q": G * d, "k": G * d, "v": H * dv}
    C = sum(sizes.values())
    names, where, w = part.layout(part.segments())
    rows = {"qkv": mat(C, width, 1.5), "a": mat(ra, width), "g": mat(rg, width, 2.0), "b": mat(H, width, 2.0)}
    stacked = torch.cat([rows[n] for n in names])
    cw = torch.randn(C, taps, generator=g) * (0.5 / taps ** 0.5)
    cw[:, -1] += 0.8
    t = {"in.weight": torch.cat([stacked, torch.zeros(w - stacked.shape[0], width)]), "o.weight": mat(width, H * dv),
         "conv.weight": cw, "a2.weight": mat(H * d, ra), "g2.weight": mat(H * dv, rg), "A_log": uni(H, -4.0, 1.0),
         "dt_bias": uni(H * d, -3.0, 0.5), "norm": uni(dv, 0.7, 1.3)}
    held = _bind(part, t, _rt(dtype))
    seg = {n: held["in.weight"][a:a + k] for n, (a, k) in where.items()}
    P = {"o": held["o.weight"], "a1": seg["a"], "g1": seg["g"], "b": seg["b"], "a2": held["a2.weight"], "g2": held["g2.weight"],
         **{n: held[n] for n in ("A_log", "dt_bias", "norm")}}
    at = 0
    for n, r in sizes.items():
        P[n], P[n + ".conv"] = seg["qkv"][at:at + r], held["conv.weight"][at:at + r]
        at += r
    return part, m, P, width


@pytest.mark.parametrize("dtype", ["float32", "bfloat16", "bfloat16-rows"])
@pytest.mark.parametrize("case", DELTA_CASES)
def test_delta_rule_part_under_every_cut(case, dtype, monkeypatch):
    """The state and the convolution's rows go from step to step in the request's slot, whatever the cut (also steps with
    fewer rows than taps).  (bfloat16 runs long portions in chunks on the tensor cores and single rows in one kernel where
    the sizes allow; "bfloat16-rows" row by row in separate kernels there too.)"""
    from atom_b200 import native
    if dtype.endswith("-rows"):
        if not native.delta_chunk_supports(case[2], case[3], torch.bfloat16):
            pytest.skip("these sizes run row by row anyway")
        monkeypatch.setattr(native, "DELTA_TC", False)
        monkeypatch.setattr(native, "DELTA_STEP", False)
        dtype = "bfloat16"
    part, m, P, W = _delta_part(case, dtype)
    lens = dict(zip("abc", case[6]))
    g = torch.Generator().manual_seed(sum(case[6]))
    x = {r: _rounded(torch.randn(n, W, generator=g), dtype) for r, n in lens.items()}
    want = {r: plain.channel_delta(x[r], P, m, EPS) for r in lens}
    for what, sched in _schedules(lens):
        h = Harness(part, dtype)
        _junk_first(h, W)
        got = h.run(x, sched)
        for r in lens:
            _close(got[r], want[r], dtype, f"{what}, request {r}", f32=5e-5, bf16=5e-2)
        assert h.manager.state_slots.num_free == 4


def _scan_inputs(n, G, H, d, dv, dtype, seed, decays=(-6.0, 1.5)):
    """(u, rn, la, beta) as delta_prepare leaves them, and the 64-bit q, k, v, g they stand for."""
    g = torch.Generator().manual_seed(seed)
    u = _rounded(torch.randn(n, 2 * G * d + H * dv, generator=g), dtype)
    heads = u[:, :2 * G * d].reshape(n, 2 * G, d)
    rn = (1.0 / torch.sqrt((heads * heads).sum(-1) + 1e-6)).float()
    rn[:, :G] *= d ** -0.5
    la = -torch.exp(torch.rand(n, H * d, generator=g) * (decays[1] - decays[0]) + decays[0])
    beta = torch.rand(n, H, generator=g)
    per = H // G
    unit = heads * rn.double()[:, :, None]
    q, k = unit[:, :G].repeat_interleave(per, 1), unit[:, G:].repeat_interleave(per, 1)
    v = u[:, 2 * G * d:].reshape(n, H, dv)
    return (u.to(_dt(dtype)), rn, la, beta), (q, k, v, torch.exp2(la.double()).view(n, H, d), beta.double())


def _scan(inputs, rows, state, cu, slots, G, H, d, dv, **kw):
    from atom_b200 import native

    u, rn, la, beta = (t[rows[0]:rows[1]].to(DEV).contiguous() for t in inputs)
    R = rows[1] - rows[0]
    out = torch.full((R, H * dv), float("nan"), dtype=torch.float32, device=DEV)
    n = native.delta_scratch_elems(R, len(slots), H, d, dv, u.dtype, max(b - a for a, b in zip(cu, cu[1:])))
    scratch = torch.full((n,), float("nan"), device=DEV) if n else None
    native.delta_scan(out, u, rn, la, beta, state, _i32(cu), _i32(slots), len(slots), G, H, d, dv, scratch=scratch,
                      max_q_len=max(b - a for a, b in zip(cu, cu[1:])), **kw)
    return out.double().cpu()


def _from_state(q, k, v, g, beta, S):
    S, out = S.double().clone(), []
    for t in range(q.shape[0]):
        S = g[t][:, :, None] * S
        w = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * w[:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out).reshape(q.shape[0], -1), S


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("decays", [(-12.0, -7.0), (-6.0, 1.5), (1.0, 6.0)])
@pytest.mark.parametrize("H,G,d,dv,T", [(4, 2, 64, 64, 333), (2, 1, 128, 128, 200), (3, 3, 12, 9, 70), (2, 2, 128, 64, 257),
                                        (2, 1, 32, 48, 130), (4, 1, 64, 128, 129), (1, 1, 96, 16, 64)])
def test_scan_of_many_rows_equals_the_scan_row_by_row(H, G, d, dv, T, decays, dtype):
    """The same rows in one step and one by one, and against the plain recurrence, with decays from almost none to a
    channel forgotten at once; requests side by side that begin with states of their own; other slots are left alone."""
    lens = [T, 1, 65]
    n = sum(lens)
    cu = [0, lens[0], lens[0] + lens[1], n]
    inputs, ref = _scan_inputs(n, G, H, d, dv, dtype, T + d, decays)
    S0 = torch.randn(4, H, d, dv, generator=torch.Generator().manual_seed(T))
    st = S0.to(DEV).contiguous()
    got = _scan(inputs, (0, n), st, cu, [2, 0, 3], G, H, d, dv)
    assert torch.equal(st[1].cpu(), S0[1])
    for slot, a, b in ((2, cu[0], cu[1]), (0, cu[1], cu[2]), (3, cu[2], cu[3])):
        want, S = _from_state(*(t[a:b] for t in ref), S0[slot])
        _close(got[a:b], want, "float32", f"slot {slot}", f32=1e-4 if dtype == "bfloat16" else 2e-5)
        _close(st[slot], S, "float32", f"state {slot}", f32=1e-4 if dtype == "bfloat16" else 2e-5)
    one = S0.to(DEV).contiguous()
    for t in range(20):
        o = _scan(inputs, (t, t + 1), one, [0, 1], [2], G, H, d, dv)
        _close(o, got[t:t + 1], "float32", f"token {t}", scale=float(got.abs().max()), f32=1e-4 if dtype == "bfloat16" else 2e-5)
    keep = S0.to(DEV).contiguous()
    again = _scan(inputs, (0, n), keep, cu, [2, 0, 3], G, H, d, dv, write_state=False)
    assert torch.equal(keep.cpu(), S0)
    _close(again, got, "float32", "without writing the state", f32=1e-6)


@pytest.mark.parametrize("lanes", [4, 8])
@pytest.mark.parametrize("d,dv", [(16, 40), (64, 24), (100, 33), (128, 64)])
def test_lanes_of_a_column_change_roundings_only(d, dv, lanes):
    inputs, ref = _scan_inputs(50, 1, 2, d, dv, "float32", d)
    st = torch.zeros(1, 2, d, dv, device=DEV)
    got = _scan(inputs, (0, 50), st, [0, 50], [0], 1, 2, d, dv, lanes=lanes)
    want, S = _from_state(*ref, torch.zeros(2, d, dv))
    _close(got, want, "float32", "outputs", f32=1e-5)
    _close(st[0], S, "float32", "state", f32=1e-5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_one_write_is_remembered_for_six_hundred_steps_and_overwritten_by_its_key(dtype):
    """One key writes a value; 600 single steps that write to orthogonal keys with no strength leave it, falling channel by
    channel as the decays say, in 32-bit whatever the activations' type; then the same key with beta 1 and another value
    replaces it (a rule that only added would hold both)."""
    H, G, d, dv, n = 2, 1, 16, 8, 600
    u = torch.zeros(n + 2, 2 * d + H * dv)
    u[:, 0] = 1.0                                          # q reads channel 0
    u[0, d], u[n + 1, d] = 1.0, 1.0                        # k: channel 0 first and last,
    u[1:n + 1, d + 5] = 1.0                                # another channel between
    u[0, 2 * d:], u[n + 1, 2 * d:] = 3.0, -1.5
    rn = torch.ones(n + 2, 2)
    la = torch.full((n + 2, H * d), -1e-3)
    la[:, d:] = -4e-3                                      # the second head forgets faster
    beta = torch.zeros(n + 2, H)
    beta[0], beta[n + 1] = 1.0, 1.0
    inputs = (u.to(_dt(dtype)), rn, la, beta)
    st = torch.zeros(2, H, d, dv, device=DEV)
    st[0] = 7.0
    outs = [_scan(inputs, (t, t + 1), st, [0, 1], [1], G, H, d, dv).view(H, dv) for t in range(n + 2)]
    for h, a in ((0, 1e-3), (1, 4e-3)):
        for t in (0, 100, n):
            want = 3.0 * 2.0 ** (-a * t)
            assert abs(float(outs[t][h, 0]) - want) < 1e-3 * want, (h, t)
    _close(outs[-1], torch.full((H, dv), -1.5, dtype=F64), "float32", "overwritten", f32=1e-5)
    assert bool((st[0] == 7.0).all())


@pytest.mark.parametrize("taps", [1, 3, 4, 9])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_what_enters_the_recurrence(taps, dtype):
    """Convolution rows from the state and the step, unit vectors (also of a head of zeros), decays without a clamp at
    either end, step sizes."""
    from atom_b200 import native

    G, H, d, dv, T = 2, 4, 8, 16, 11
    dt = _dt(dtype)
    C = 2 * G * d + H * dv
    g = torch.Generator().manual_seed(taps)
    hist = _rounded(torch.randn(taps - 1 + T, C, generator=g), dtype)
    hist[:, :d] = 0.0                                      # the first query head is zero
    w = _rounded(torch.randn(C, taps, generator=g), dtype)
    z = torch.randn(T, H * d, generator=g) * 3
    z[0, :6] = torch.tensor([-200.0, -30.0, 0.0, 20.0, 90.0, 300.0])
    A, b = (_rounded(torch.randn(k, generator=g), dtype) for k in (H, H * d))
    raw = _rounded(torch.randn(T, H, generator=g) * 4, dtype)
    state = torch.zeros(3, max(taps - 1, 1), C, dtype=dt)
    state[2, :taps - 1] = hist[:taps - 1].to(dt)
    dev = lambda t: t.to(dt).to(DEV).contiguous()
    u = torch.empty(T, C, dtype=dt, device=DEV)
    rn, beta, la = torch.empty(T, 2 * G, device=DEV), torch.empty(T, H, device=DEV), z.to(DEV).contiguous()
    native.delta_prepare(u, rn, dev(hist[taps - 1:]), dev(w), state.to(DEV) if taps > 1 else None, la, dev(A), dev(b), dev(raw),
                         beta, _i32([0] * T), _i32([0, T]), _i32([2]), G, H, d, dv, 0.5, 1e-6)
    want = plain.silu(plain.causal_conv(hist, w))[taps - 1:]
    _close(u, want, dtype, "u", f32=2e-6, bf16=5e-3)
    heads = u.double().cpu()[:, :2 * G * d].reshape(T, 2 * G, d)
    f = 1.0 / torch.sqrt((heads * heads).sum(-1) + 1e-6)
    f[:, :G] *= 0.5
    assert torch.allclose(rn.double().cpu(), f, rtol=1e-5)
    zz = z.double() + b
    sp = torch.log1p(torch.exp(-zz.abs())) + zz.clamp(min=0)
    ref = -torch.exp(A).repeat_interleave(d)[None] * sp / np.log(2.0)
    assert torch.allclose(la.double().cpu(), ref, rtol=2e-6, atol=1e-30)
    assert torch.allclose(beta.double().cpu(), torch.sigmoid(raw), rtol=2e-6)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("gate", ["silu", "sigmoid"])
@pytest.mark.parametrize("H,dv", [(5, 24), (9, 128), (3, 50), (2, 136), (8, 100)])
def test_output_norm_per_head_with_its_gate(H, dv, gate, dtype):
    from atom_b200 import native

    T = 7
    dt = _dt(dtype)
    g = torch.Generator().manual_seed(3)
    o = torch.randn(T, H * dv, generator=g)
    z = _rounded(torch.randn(T, H * dv + 8, generator=g) * 2, dtype)
    w = _rounded(torch.rand(dv, generator=g) + 0.5, dtype)
    wide = torch.full((T, H * dv + 16), 9.0, dtype=dt, device=DEV)
    native.gla_gate_norm(wide[:, 8:8 + H * dv], o.to(DEV), z.to(dt).to(DEV)[:, 4:4 + H * dv], w.to(dt).to(DEV), 1e-4, H, dv,
                         _i32([0] * T), gate, 0.75)
    zz = z[:, 4:4 + H * dv]
    act = torch.sigmoid(zz) * (zz if gate == "silu" else 1.0)
    want = (plain.rms(o.double().view(T, H, dv), 1e-4) * w).reshape(T, -1) * act * 0.75
    _close(wide[:, 8:8 + H * dv], want, dtype, gate, f32=2e-6, bf16=6e-3)
    assert bool((wide[:, :8] == 9).all()) and bool((wide[:, 8 + H * dv:] == 9).all())


# ============================================================================= differential attention

ATT_CASES = [  # H, G, dk, dv, rot (base, dims), chunk, diff, page, lens
    (4, 2, 16, 24, (10000.0, 8), 24, 0.35, 16, (70, 9, 41)),
    (2, 1, 24, 16, None, None, 0.2, 8, (50, 3, 27)),
    (3, 3, 8, 40, (77.0, 4), 7, 0.6, 8, (40, 17, 2)),
    (5, 5, 20, 12, (1000.0, 12), 1, 0.45, 16, (33, 5, 20)),
    (6, 1, 12, 28, (300.0, 6), 33, 0.1, 16, (90, 48, 7)),
    (8, 2, 64, 128, (100000.0, 64), None, 0.5, 32, (300, 40, 131)),
    (4, 4, 32, 128, (10000.0, 32), 64, 0.7, 16, (150, 70, 4)),
    (8, 1, 128, 128, (1000000.0, 128), 50, 0.3, 16, (140, 60, 10)),
    (6, 2, 80, 48, (10000.0, 40), 17, 0.4, 8, (64, 65, 63)),
    (3, 1, 7, 5, (50.0, 6), None, 0.25, 8, (30, 2, 11)),
    (12, 3, 48, 16, (300.0, 16), 129, 0.8, 16, (270, 20, 5)),
]


def _attention_args(case, width, **over):
    from atom_b200.parts.spec import PartSpec

    H, G, dk, dv, rot, chunk, diff, page, lens = case
    position = PartSpec("rope_yarn", {"rotary_dim": rot[1], "theta": rot[0]}) if rot else None
    return dict(dict(hidden_size=width, num_heads=H, num_kv_heads=G, key_dim=dk, value_dim=dv, scale=1.7 / dk ** 0.5, diff=diff,
                     norm_eps=EPS, position=position, chunk=chunk, held=(chunk, True) if chunk else None), **over)


def _attention_part(case, dtype, width=72, seed=0, own=True, **over):
    H, G, dk, dv, rot, chunk, diff, page, lens = case
    args = _attention_args(case, width, own_keys=own, **over)
    part = _part("mixer", "differential_attention", **args)
    m = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": args["scale"], "diff": diff}
    if rot:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    if args["chunk"]:
        m["mask"] = {"size": args["chunk"]}
    g = torch.Generator().manual_seed(H * dk + dv + seed)
    mat = lambda o, gain=1.0: torch.randn(o, width, generator=g) * gain / width ** 0.5
    sizes = {"q": 2 * H * dk, "k": 2 * G * dk, "v": G * dv} if own else {"q": 2 * H * dk}
    pad = part.params()["in.weight"].pad
    t = {"in.weight": torch.cat([mat(r, 1.5) for r in sizes.values()] + [torch.zeros(pad, width)]),
         "o.weight": torch.randn(width, H * dv, generator=g) / (H * dv) ** 0.5,
         "lambdas": torch.randn(4, dk, generator=g) * (0.5 / dk ** 0.5), "q_norm": torch.rand(dk, generator=g) + 1.0}
    if own:
        t["k_norm"] = torch.rand(dk, generator=g) + 1.0
    held = _bind(part, t, _rt(dtype))
    P = {"o": held["o.weight"], "q.norm": held["q_norm"], **dict(zip(("lq1", "lk1", "lq2", "lk2"), held["lambdas"]))}
    if own:
        P["k.norm"] = held["k_norm"]
    at = 0
    for n, r in sizes.items():
        P[n] = held["in.weight"][at:at + r]
        at += r
    return part, m, P, width


def _tc_off(case, dtype, monkeypatch):
    from atom_b200 import native
    if not dtype.endswith("-plain"):
        return dtype
    if not native.window_attention_tc_supports(case[2], case[3], torch.bfloat16, 2):
        pytest.skip("these sizes run the plain kernel anyway")
    monkeypatch.setattr(native, "WINDOW_TC", False)
    return "bfloat16"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16", "bfloat16-plain"])
@pytest.mark.parametrize("case", ATT_CASES)
def test_differential_attention_part_under_every_cut(case, dtype, monkeypatch):
    """(bfloat16 runs the tensor-core kernel where it takes the sizes; "bfloat16-plain" the plain kernel there too.)"""
    dtype = _tc_off(case, dtype, monkeypatch)
    part, m, P, W = _attention_part(case, dtype)
    page, lens = case[7], dict(zip("abc", case[8]))
    g = torch.Generator().manual_seed(sum(case[8]))
    x = {r: _rounded(torch.randn(n, W, generator=g), dtype) for r, n in lens.items()}
    want = {r: plain.differential_attention(x[r], P, m, EPS, plain.keys_and_values(x[r], P, m, EPS)) for r in lens}
    for what, sched in _schedules(lens):
        h = Harness(part, dtype, page=page, pages=3 * (max(lens.values()) // page + 3))
        _junk_first(h, W)
        got = h.run(x, sched)
        for r in lens:
            _close(got[r], want[r], dtype, f"{what}, request {r}", f32=5e-5, bf16=5e-2)
        assert all(gr.pool.num_used == 0 for gr in h.manager.groups) and h.manager.state_slots.num_free == 4


class _OwnerThenReader:
    """Two mixers on one cache slot, as two layers are: the reader sees the owner's keys of this step and of earlier
    ones and writes nothing."""

    def __init__(self, owner, reader):
        self.owner, self.reader = owner, reader

    def cache_need(self):
        assert self.owner.cache_need() == self.reader.cache_need()
        return self.owner.cache_need()

    def forward(self, x, step, cache, writes_cache):
        self.owner.forward(x, step, cache, writes_cache)
        before = cache.k_pages.clone(), cache.v_pages.clone()
        y = self.reader.forward(x.flip(1).contiguous(), step, cache, False)
        assert torch.equal(before[0], cache.k_pages) and torch.equal(before[1], cache.v_pages)
        return y


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case,readers_chunk,readers_heads", [(ATT_CASES[0], 40, 6), (ATT_CASES[1], 9, 3), (ATT_CASES[6], 64, 8),
                                                              (ATT_CASES[8], None, 2), (ATT_CASES[5], 100, 2)])
def test_keys_and_values_of_another_layer(case, readers_chunk, readers_heads, dtype):
    """The reader has other inputs, queries, head count, chunks, diff and lambdas; the pages are held as far back as
    either of the two looks."""
    chunks = [case[5], readers_chunk]
    held = None if None in chunks else (max(chunks), chunks[0] == chunks[1])
    owner, mo, Po, W = _attention_part(case, dtype, held=held)
    other = (readers_heads,) + case[1:5] + (readers_chunk, 0.55) + case[7:]
    reader, mr, Pr, _ = _attention_part(other, dtype, seed=9, own=False, held=held)
    page, lens = case[7], dict(zip("abc", case[8]))
    g = torch.Generator().manual_seed(sum(case[8]))
    x = {r: _rounded(torch.randn(n, W, generator=g), dtype) for r, n in lens.items()}
    want = {r: plain.differential_attention(x[r].flip(1), Pr, mr, EPS, plain.keys_and_values(x[r], Po, mo, EPS)) for r in lens}
    for what, sched in _schedules(lens):
        h = Harness(_OwnerThenReader(owner, reader), dtype, page=page, pages=3 * (max(lens.values()) // page + 3))
        _junk_first(h, W)
        got = h.run(x, sched)
        for r in lens:
            _close(got[r], want[r], dtype, f"{what}, request {r}", f32=5e-5, bf16=5e-2)


def _kernels(dk, dv, dtype, maps=2):
    from atom_b200 import native
    return ["plain", "tc1", "tc3", "tc7"] if native.window_attention_tc_supports(dk, dv, _dt(dtype), maps) else ["plain"]


def _run_attention(q, k, v, scale, chunk, maps, out_scale, dtype, page, cuts, kernel, gate=None):
    """One request's keys and values in scrambled pages, the queries in portions ``cuts``; q [T, H, 2, dk], k [T, G, 2, dk]
    (or without the maps' axis for maps None); the output is a part of wider rows (the rest must stay as it was)."""
    from atom_b200 import native

    T, H, G, dk, dv = q.shape[0], q.shape[1], k.shape[1], q.shape[-1], v.shape[2]
    n_maps = 2 if maps else 1
    dt = _dt(dtype)
    table, kp, _ = _win_pages(T, G * n_maps, page, dk, dv, dtype, seed=T)
    _, _, vp = _win_pages(T, G, page, dk, dv, dtype, seed=T)
    out = torch.zeros(T, H * dv, dtype=dt, device=DEV)
    at = 0
    for n in cuts:
        n = min(n, T - at)
        if n <= 0:
            continue
        j = torch.arange(at, at + n, device=DEV)
        pg = table[0].long()[j // page]
        kp[pg, :, j % page] = k[at:at + n].reshape(n, G * n_maps, dk).to(dt).to(DEV)
        vp[pg, :, j % page] = v[at:at + n].to(dt).to(DEV)
        wide = torch.full((n, H * dv + 16), 9.0, dtype=dt, device=DEV)
        o = wide[:, 8:8 + H * dv]
        qd = q[at:at + n].reshape(n, -1).to(dt).to(DEV).contiguous()
        kw = dict(out_scale=out_scale, chunked=bool(chunk), maps=maps, gate=None if gate is None else gate[at:at + n].to(dt).to(DEV))
        if kernel.startswith("tc"):
            ns = int(kernel[2:])
            scratch = torch.full((native.attention_mixed_scratch_elems(n, H * n_maps, dv, ns),), float("nan"), device=DEV) if ns > 1 else None
            native.window_attention_tc(o, qd, kp, vp, table, _i32(range(at, at + n)), _i32([0] * n), _i32([0, n]), 1, H, G, dk, dv,
                                       scale, 0.0, chunk, 0, ns, scratch, heads_rows=(n == 1 and at % 2 == 0), **kw)
        else:
            native.window_attention(o, qd, kp, vp, table, _i32(range(at, at + n)), _i32([0] * n), H, G, dk, dv, scale, 0.0, chunk,
                                    0, **kw)
        assert bool((wide[:, :8] == 9).all()) and bool((wide[:, 8 + H * dv:] == 9).all())
        out[at:at + n] = o
        at += n
    assert at == T
    return out.double().cpu().view(T, H, dv)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk", [1, 2, 16, 17, 64, 65, 100, 300, 0])
def test_single_keys_at_the_chunks_borders(chunk, dtype):
    """A key row that carries a mark only it has and a score far above all others, once in the first map and once in the
    second: seen from every later place of its chunk and from no place of the next one, in a prompt, across portions that
    end at every place around the border and decoded one by one.  The keys stand first, last and in the middle of a chunk."""
    H, G, dk, dv, page, T = 4, 2, 32, 16, 16, 330
    lam, eps = 0.5, 1e-5
    c = chunk or 1000
    marks = sorted({95 // c * c, min(95 // c * c + c - 1, 130), min(95 // c * c + (c - 1) // 2, 140)})
    for needle in marks:
        for which in (0, 1):
            g = torch.Generator().manual_seed(chunk + needle)
            k = torch.randn(T, G, 2, dk, generator=g) * 0.1
            v = torch.randn(T, G, dv, generator=g) * 0.1
            q = torch.randn(T, H, 2, dk, generator=g) * 0.1
            v[:, :, 0], k[..., 0], q[..., 0] = 0.0, 0.0, 3.0
            v[needle, :, 0], k[needle, :, which, 0] = 1.0, 4.0          # a score of 12 against a few tenths
            q, k, v = _rounded(q, dtype), _rounded(k, dtype), _rounded(v, dtype)
            a = [plain.softmax_attention(q[:, :, i], k[:, :, i], v, 1.0, chunk or None) for i in (0, 1)]
            want = plain.rms(a[0] - lam * a[1], eps) * 0.7
            sees = lambda i: i >= needle and i // c == needle // c
            for i in range(T):
                assert (float(a[which][i, 0, 0]) > 0.9) == sees(i)
            edge = min((needle // c + 1) * c, T - 3)
            cut_sets = [[T], [edge - 1, 1, 1, 1, T], [edge, T], [edge + 1, T], [needle, 2, min(c, 60), 2, T]]
            if 0 < chunk <= 65:
                cut_sets.append([needle + 1] + [1] * min(2 * chunk + 3, T - needle - 1) + [T])
            for cuts in cut_sets:
                for kernel in _kernels(dk, dv, dtype):
                    if kernel in ("tc3", "tc7") and len(cuts) > 20:
                        continue
                    got = _run_attention(q, k, v, 1.0, chunk, (lam, eps), 0.7, dtype, page, cuts, kernel)
                    what = f"{kernel}, chunk {chunk}, key {needle} of map {which + 1}, cuts {cuts[:4]}"
                    assert all((float(got[i, 0, 0]) != 0) == sees(i) for i in range(T)), what
                    _close(got, want, dtype, what, f32=3e-5, bf16=2e-2)


@pytest.mark.parametrize("maps", [None, (0.65, 1e-5), (-0.3, 1e-3)])
@pytest.mark.parametrize("H,G,dk,dv,chunk,page,T", [(8, 2, 64, 128, 0, 32, 333), (12, 3, 96, 32, 100, 16, 300),
                                                     (4, 1, 128, 128, 70, 16, 270), (3, 3, 48, 16, 65, 8, 200),
                                                     (16, 1, 16, 64, 33, 16, 150)])
def test_tensor_core_attention_in_chunks_against_plain(H, G, dk, dv, chunk, page, T, maps):
    """One map or two, with a gate per head beside them."""
    n_maps = 2 if maps else 1
    g = torch.Generator().manual_seed(T + dk)
    q, k = (_rounded(torch.randn(T, n, n_maps, dk, generator=g), "bfloat16") for n in (H, G))
    v = _rounded(torch.randn(T, G, dv, generator=g), "bfloat16")
    gate = _rounded(torch.randn(T, H, generator=g) * 2, "bfloat16")
    scale = 3.0 / dk ** 0.5
    a = [plain.softmax_attention(q[:, :, i], k[:, :, i], v, scale, chunk or None) for i in range(n_maps)]
    want = (plain.rms(a[0] - maps[0] * a[1], maps[1]) if maps else a[0]) * torch.sigmoid(gate)[:, :, None]
    kernels = _kernels(dk, dv, "bfloat16", n_maps)
    assert "tc1" in kernels
    for kernel in kernels:
        for cuts in ([T], [T - 9] + [1] * 9, [13, 64, 5, 2, 129, 2, 70, 3, 17] * 8):
            got = _run_attention(q, k, v, scale, chunk, maps, 1.0, "bfloat16", page, cuts, kernel, gate)
            _close(got, want, "bfloat16", f"{kernel}, cuts {cuts[:3]}", bf16=1.5e-2)


# ============================================================================= feed-forwards

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("W,ff,limit,T", [(64, 72, 1.2, 5), (256, 512, 0.7, 40), (100, 30, 2.0, 17), (256, 1024, 1.5, 700)])
def test_dense_feed_forward_with_clamps(W, ff, limit, T, dtype):
    from types import SimpleNamespace

    part = _part("ffn", "gated_clamped", hidden_size=W, intermediate_size=ff, limit=limit)
    g = torch.Generator().manual_seed(W + ff)
    mat = lambda o, i, gain=1.5: torch.randn(o, i, generator=g) * gain / i ** 0.5
    held = _bind(part, {"gate_up.weight": torch.cat([mat(ff, W), mat(ff, W)]), "down.weight": mat(W, ff)}, _rt(dtype))
    P = {"gate": held["gate_up.weight"][:ff], "up": held["gate_up.weight"][ff:], "down": held["down.weight"]}
    x = _rounded(torch.randn(T, W, generator=g), dtype)
    got = part.forward(x.to(_dt(dtype)).to(DEV), SimpleNamespace())
    _close(got, plain.clamped_mlp(x, P, "", limit), dtype, "dense", f32=2e-5, bf16=2e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("W,E,top,ff,limit,shared,factor,T", [
    (64, 6, 2, 24, 1.1, (40, 0.8), 1.7, 45), (96, 5, 3, 40, 2.0, None, 1.0, 33), (100, 3, 3, 28, 0.7, (36, 2.5), 0.4, 7),
    (72, 1, 1, 16, 1.0, (8, 0.5), 1.0, 1), (128, 16, 4, 64, 1.5, (64, 1.0), 2.0, 300)])
def test_experts_with_renormalised_sigmoid_scores_and_a_gated_shared_one(W, E, top, ff, limit, shared, factor, T, dtype):
    from types import SimpleNamespace

    part = _part("ffn", "routed_experts", hidden_size=W, num_experts=E, top=top, intermediate_size=ff,
                 shared_size=shared[0] if shared else None, score="sigmoid", renormalize=True, weight_on="output",
                 shared_gate=shared is not None, factor=factor, sum_eps=1e-20, limit=limit, shared_limit=shared[1] if shared else None)
    g = torch.Generator().manual_seed(W + E)
    mat = lambda o, i, gain=1.5: torch.randn(o, i, generator=g) * gain / i ** 0.5
    t = {"router.weight": torch.cat([mat(E, W, 2.0), mat(1, W)] if shared else [mat(E, W, 2.0)]),
         "gate_up.weight": torch.cat([mat(ff, W) for _ in range(2 * E)]), "down.weight": torch.cat([mat(W, ff) for _ in range(E)])}
    if shared:
        t["shared.gate_up.weight"], t["shared.down.weight"] = mat(2 * shared[0], W), mat(W, shared[0])
    held = _bind(part, t, _rt(dtype))
    P = {"router": held["router.weight"][:E], "shared.sg": held["router.weight"][E:]}
    for e in range(E):
        P[f"e{e}.gate"] = held["gate_up.weight"][2 * e * ff:(2 * e + 1) * ff]
        P[f"e{e}.up"] = held["gate_up.weight"][(2 * e + 1) * ff:(2 * e + 2) * ff]
        P[f"e{e}.down"] = held["down.weight"][e * W:(e + 1) * W]
    mlp = {"router": {"top": top, "scale": factor}, "expert": {"limit": limit}}
    if shared:
        S = shared[0]
        P["shared.gate"], P["shared.up"] = held["shared.gate_up.weight"][:S], held["shared.gate_up.weight"][S:]
        P["shared.down"], mlp["shared"] = held["shared.down.weight"], {"limit": shared[1]}
    x = _rounded(torch.randn(T, W, generator=g), dtype)
    want = plain.expert_mixture(x, P, mlp)
    s = torch.sigmoid(x @ P["router"].T).sort(-1, descending=True).values
    clear = (s[:, top - 1] - s[:, top] > 2e-3) if top < E else torch.ones(T, dtype=torch.bool)
    assert clear.double().mean() > 0.8
    step = SimpleNamespace(seq_of_token=_i32([0] * T), num_tokens=T, num_seqs=1)
    for _ in range(2):                        # twice: what the first call leaves in the workspace does not leak
        got = part.forward(x.to(_dt(dtype)).to(DEV), step)
        _close(got.cpu()[clear], want[clear], dtype, "experts", f32=3e-5, bf16=3e-2)


# ============================================================================= whole models

LENGTHS = {"A": [1, 2, 9, 41, 100, 70], "B": [3, 17, 64, 131, 30], "C": [5, 33, 90, 48, 70], "D": [4, 70, 230, 33],
           "E": [3, 40, 75, 1, 20]}


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    out = {}
    for name, cfg in tv.CONFIGS.items():
        d = str(tmp_path_factory.mktemp(f"vunepel_{name}"))
        tv.write_model(cfg, d, tv.SEEDS[name])
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
@pytest.mark.parametrize("name", list(tv.CONFIGS))
def test_layer_by_layer_against_plain(dirs, name, dtype):
    """The residual stream after every layer of a short prompt (what the next norm reads)."""
    from atom_b200.engine.batch import StepEntry
    from atom_b200.parts.linear import SumDelta
    cfg, w = tv.read_model(dirs[name])
    p = tv.prompts(tv.CONFIGS[name], [45], seed=2)[0]
    want = plain.forward(cfg, w, p, return_layers=True)[1]
    runner = _runner(dirs[name], dtype, 64, tv.PAGE[name])
    seen = []
    for b in runner.model.blocks:
        def run(residual, delta, step, cache, wc, _o=b.run):
            out = _o(residual, delta, step, cache, wc)
            added = (out.a.double() + out.b.double()) if isinstance(out, SumDelta) else out.double()
            seen.append(residual.double() + added)
            return out
        b.run = run
    runner.step([StepEntry("a", p, [0])])
    runner.check_status()
    assert len(seen) == len(want) == len(cfg["layers"])
    for i, (g, r) in enumerate(zip(seen, want)):
        _close(g, r, dtype, f"after layer {i}", f32=3e-5, bf16=3e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(tv.CONFIGS))
def test_every_cut_matches_plain(dirs, name, dtype):
    """Whole; the last 48 tokens one by one (chunks end among them); portions of changing size down to two tokens; pairs of
    tokens throughout; up to four live requests with portions beside single tokens in a pool so small that pages and state
    slots are used again."""
    seqs = _seqs(name)
    ref = _plain_logits(dirs[name], seqs)
    mixed, peak = traces.mixed(seqs, max_live=4, budget_tokens=320)
    assert peak <= 320
    runner = _runner(dirs[name], dtype, 320, tv.PAGE[name], max_num_seqs=4)
    for what, steps in (("whole", traces.whole(seqs)), ("tail", traces.tail_by_token(seqs, 48)),
                        ("ragged", traces.ragged(seqs)), ("pairs", traces.ragged(seqs, sizes=(2,))), ("mixed", mixed)):
        if what == "pairs":
            steps = [s for s in steps if s["entries"][0]["id"] in ("r1", "r2")]       # (two requests are enough)
            sub = {r: ref[r] for r in ("r1", "r2")}
            _compare(traces.collect(steps, _replay(runner, steps)), sub, dtype, f"{name}/{what}")
            continue
        _compare(traces.collect(steps, _replay(runner, steps)), ref, dtype, f"{name}/{what}")
        assert all(g.pool.num_used == 0 for g in runner.cache.groups) and runner.cache.state_slots.num_free == 4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_request_freed_half_way_and_fed_again(dirs, name, dtype):
    """What preemption by recomputation does: pages and the state slot go back, another request takes them, and the
    victim starts over on whatever slot is free, with a state and convolution rows of zeros."""
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
    from atom_b200.engine.batch import StepEntry

    name = "D"
    ps = tv.prompts(tv.CONFIGS[name], [150, 3, 27, 64], seed=99)
    runner = _runner(dirs[name], dtype, 1024, tv.PAGE[name])
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
    """300 tokens decoded one by one after a prompt of three: pages fill, follow one another and are given back as chunks
    end; the recurrent state and the convolution's rows are read and written 300 times."""
    seqs = {"long": tv.prompts(tv.CONFIGS[name], [303], seed=4)[0]}
    ref = _plain_logits(dirs[name], seqs)
    steps = traces.tail_by_token(seqs, 300)
    runner = _runner(dirs[name], dtype, 304, tv.PAGE[name])
    _compare(traces.collect(steps, _replay(runner, steps)), ref, dtype, "long decoding")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "D"])
def test_captured_steps_match_plain(dirs, name, dtype):
    """Decode steps and small mixed steps replayed from CUDA graphs, with padding rows and padding requests."""
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


@pytest.mark.parametrize("name,chunk", [("A", 8), ("C", 13), ("E", 5)])
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
def test_trace_run_program_on_a_vunepel_folder(dirs, tmp_path, dtype):
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
