"""Vudezen: a decoder-only model whose layers are listed one by one in config.json.  Every sub-block has a layer norm before
and after it and enters the residual stream times a constant; the mixer is attention with a sink and a gate per head (all
earlier tokens, rotary positions on neighbouring pairs with YaRN's stretch, values blended with the first such layer's),
or two mixers side by side whose outputs are added with a factor each: attention of that kind over a sliding window, and
a state-space recurrence (Mamba-2).  The feed-forward is a mixture of experts with clamped gates, grouped choice and
identity experts beside a shared expert, or absent.

config.json:  ``architecture`` "Vudezen"; ``vocab``, ``width``; ``norm.eps``; ``residual_mult``; ``logit_scale``,
``logit_softcap`` (absent or 0: none);
``layers``: entries with ``type`` ("parallel" | "attention"), ``mixer``, ``mlp`` (or null)
  attention mixer: heads, kv_heads, dim, vdim, scale, rot {base, dims, scaling {factor, original, fast, slow}} (absent: no
      rotation; scaling absent: plain frequencies), mask {size} (absent: every earlier token is seen), v_mix (absent: false)
  parallel mixer:  left (as an attention mixer), left_scale, right {heads, vdim, state, groups, conv (taps), norm_groups},
      right_scale
  mlp: {kind "moe", router {experts, top, identity (absent: 0), groups {count, keep} (absent: none), scale},
      expert {ff, limit}, shared {ff, limit} (absent: none)}

Tensors: ``embed``, ``head``, ``final.norm``, per layer ``l<i>.norm1``, ``norm1b``, ``norm2``, ``norm2b`` (every norm with a
bias ``<name>.b``) and
  attention: ``l<i>.mix.{q,k,v,o}`` with ``.b`` each, ``l<i>.mix.{sink,g}``, with v_mix ``l<i>.mix.vmix`` (a single number)
  parallel:  ``l<i>.mix.left.{q,k,v}`` with ``.b`` each, ``l<i>.mix.left.{sink,g,o}``,
             ``l<i>.mix.right.{in,conv,conv.b,dt_bias,A_log,D,norm,o}``
  moe:       ``l<i>.mlp.{router,correction}``, ``l<i>.mlp.e<j>.{gate,up,down}``, ``l<i>.mlp.shared.{gate,up,down}``
Matrices are [out, in].

  x = embed[token]
  per layer:  x += m norm(mixer(norm(x; norm1)); norm1b);   x += m norm(mlp(norm(x; norm2)); norm2b)   (if it has one)
  logits = cap tanh(logit_scale (head norm(x; final.norm)) / cap)
The mixers' formulas stand in parts/sink_attention.py, parts/ssm.py and parts/summed_mixers.py, the feed-forward's in
parts/moe.py (routed_experts).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, ClassVar, Dict, Mapping, Optional, Tuple

from ..config.model_config import ConfigError, ModelConfig, cfg_get, cfg_positive
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunEntry
from ..parts.summed_mixers import projected_spec, summed_mixers_spec
from .registry import register_architecture

# Nothing in the design bounds a position (angles are computed from the position itself); a request's length is
# bounded by the engine's max_model_len, which defaults to this many tokens.
_DEFAULT_MAX_LEN = 32768
_MAX_POSITION = 1 << 24        # positions are exact in 32-bit floats up to here

_SUM_EPS = 1e-20               # added to the sum that the chosen experts' scores are divided by


@dataclass(frozen=True)
class Attention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: Optional[float]
    rot_dims: int
    rot_scaling: Optional[Tuple[float, float, float, float]]     # factor, original, fast, slow
    window: Optional[int]
    v_mix: bool


@dataclass(frozen=True)
class StateSpace:
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_groups: int


@dataclass(frozen=True)
class Pair:
    left: Attention
    left_scale: float
    right: StateSpace
    right_scale: float


@dataclass(frozen=True)
class Experts:
    experts: int
    identity: int
    top: int
    groups: Optional[Tuple[int, int]]      # count, keep
    scale: float
    ff: int
    limit: float
    shared: Optional[Tuple[int, float]]    # ff, limit


@dataclass(frozen=True)
class VudezenLayer:
    type: str
    mixer: Any                       # Attention | Pair
    moe: Optional[Experts]           # None: no feed-forward


def _obj(d: Mapping, key: str, where: str) -> Mapping:
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}'{key}' must be an object")
    return v


def _number(d: Mapping, key: str, where: str) -> float:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"config.json: {where}'{key}' must be a number, got {v!r}")
    return float(v)


def _positive(d: Mapping, key: str, where: str) -> float:
    v = _number(d, key, where)
    if v <= 0:
        raise ConfigError(f"config.json: {where}{key} must be positive, got {v}")
    return v


def _count(d: Mapping, key: str, where: str, least: int = 1) -> int:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, int) or v < least:
        raise ConfigError(f"config.json: {where}'{key}' must be an int >= {least}, got {v!r}")
    return v


def _attention(m: Mapping, w: str) -> Attention:
    base, dims, scaling, window = None, 0, None, None
    if m.get("rot") is not None:
        rot = _obj(m, "rot", w)
        base, dims = _number(rot, "base", w + "rot."), _count(rot, "dims", w + "rot.", 0)
        if base <= 1.0:
            raise ConfigError(f"config.json: {w}rot.base must exceed 1, got {base}")
        if rot.get("scaling") is not None:
            sc = _obj(rot, "scaling", w + "rot.")
            scaling = tuple(_positive(sc, k, w + "rot.scaling.") for k in ("factor", "original", "fast", "slow"))
    if m.get("mask") is not None:
        window = _count(_obj(m, "mask", w), "size", w + "mask.")
    v_mix = m.get("v_mix", False)
    if not isinstance(v_mix, bool):
        raise ConfigError(f"config.json: {w}v_mix must be true or false, got {v_mix!r}")
    out = Attention(heads=_count(m, "heads", w), kv_heads=_count(m, "kv_heads", w), dim=_count(m, "dim", w),
                    vdim=_count(m, "vdim", w), scale=_number(m, "scale", w), rot_base=base, rot_dims=dims,
                    rot_scaling=scaling, window=window, v_mix=v_mix)
    if out.heads % out.kv_heads:
        raise ConfigError(f"config.json: {w}heads ({out.heads}) must be a multiple of kv_heads ({out.kv_heads})")
    if out.rot_dims % 2 or out.rot_dims > out.dim:
        raise ConfigError(f"config.json: {w}rot.dims ({out.rot_dims}) must be even and at most dim ({out.dim})")
    return out


def _pair(m: Mapping, w: str) -> Pair:
    r, wr = _obj(m, "right", w), w + "right."
    right = StateSpace(heads=_count(r, "heads", wr), vdim=_count(r, "vdim", wr), state=_count(r, "state", wr),
                       groups=_count(r, "groups", wr), taps=_count(r, "conv", wr), norm_groups=_count(r, "norm_groups", wr))
    if right.heads % right.groups:
        raise ConfigError(f"config.json: {wr}heads ({right.heads}) must be a multiple of groups ({right.groups})")
    if (right.heads * right.vdim) % right.norm_groups:
        raise ConfigError(f"config.json: {wr}norm_groups ({right.norm_groups}) must divide heads * vdim")
    left = _attention(_obj(m, "left", w), w + "left.")
    if left.v_mix:
        raise ConfigError(f"config.json: {w}left.v_mix: only an 'attention' layer blends values")
    return Pair(left=left, left_scale=_number(m, "left_scale", w), right=right, right_scale=_number(m, "right_scale", w))


def _mlp(mlp, w: str) -> Optional[Experts]:
    if mlp is None:
        return None
    if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
        raise ConfigError(f"config.json: {w}mlp must be null or an object of kind 'moe'")
    w += "mlp."
    r, e = _obj(mlp, "router", w), _obj(mlp, "expert", w)
    groups = None
    if r.get("groups") is not None:
        g = _obj(r, "groups", w + "router.")
        groups = (_count(g, "count", w + "router.groups."), _count(g, "keep", w + "router.groups."))
    shared = None
    if mlp.get("shared") is not None:
        s = _obj(mlp, "shared", w)
        shared = (_count(s, "ff", w + "shared."), _positive(s, "limit", w + "shared."))
    out = Experts(experts=_count(r, "experts", w + "router."),
                  identity=_count(r, "identity", w + "router.", 0) if r.get("identity") is not None else 0,
                  top=_count(r, "top", w + "router."), groups=groups,
                  scale=_number(r, "scale", w + "router.") if r.get("scale") is not None else 1.0,
                  ff=_count(e, "ff", w + "expert."), limit=_positive(e, "limit", w + "expert."), shared=shared)
    n = out.experts + out.identity
    if groups is not None and (n % groups[0] or groups[1] > groups[0]):
        raise ConfigError(f"config.json: {w}router.groups: {groups[1]} of {groups[0]} equal groups of {n} experts")
    if out.top > (n if groups is None else groups[1] * (n // groups[0])):
        raise ConfigError(f"config.json: {w}router.top ({out.top}) exceeds the experts that can be chosen")
    return out


@dataclass(frozen=True)
class VudezenConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm_eps: float = 0.0
    residual_mult: float = 1.0
    logit_scale: float = 1.0
    logit_softcap: Optional[float] = None
    layers: Tuple[VudezenLayer, ...] = ()

    ARCHITECTURE: ClassVar[str] = "Vudezen"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "VudezenConfig":
        entries = d.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, e in enumerate(entries):
            w = f"layers[{i}]."
            if not isinstance(e, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = e.get("type")
            m = _obj(e, "mixer", w)
            if kind == "attention":
                mixer = _attention(m, w + "mixer.")
            elif kind == "parallel":
                mixer = _pair(m, w + "mixer.")
            else:
                raise ConfigError(f"config.json: {w}type {kind!r} is not supported (parallel, attention)")
            layers.append(VudezenLayer(kind, mixer, _mlp(e.get("mlp"), w)))
        mixing = {(L.mixer.kv_heads, L.mixer.vdim) for L in layers if L.type == "attention" and L.mixer.v_mix}
        if len({g * v for g, v in mixing}) > 1:
            raise ConfigError("config.json: layers with v_mix must have values of one size")
        cap = d.get("logit_softcap")
        if cap is not None:
            cap = _number(d, "logit_softcap", "")
            if cap < 0:
                raise ConfigError(f"config.json: logit_softcap must be positive, got {cap}")
            cap = cap or None                            # (0 stands for no cap, as an absent key does)
        return cls(architecture=cls.ARCHITECTURE, vocab=cfg_positive("vocab", cfg_get(d, "vocab", int)),
                   width=cfg_positive("width", cfg_get(d, "width", int)),
                   norm_eps=_positive(_obj(d, "norm", ""), "eps", "norm."),
                   residual_mult=_number(d, "residual_mult", "") if d.get("residual_mult") is not None else 1.0,
                   logit_scale=_number(d, "logit_scale", "") if d.get("logit_scale") is not None else 1.0,
                   logit_softcap=cap, layers=tuple(layers))

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                               "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult,
                               "logit_scale": self.logit_scale, "layers": []}
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap

        def attention(a: Attention) -> dict:
            m: Dict[str, Any] = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale}
            if a.rot_base is not None:
                m["rot"] = {"base": a.rot_base, "dims": a.rot_dims}
                if a.rot_scaling is not None:
                    m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), a.rot_scaling))
            if a.window is not None:
                m["mask"] = {"size": a.window}
            if a.v_mix:
                m["v_mix"] = True
            return m

        for L in self.layers:
            if L.type == "attention":
                mixer = attention(L.mixer)
            else:
                r = L.mixer.right
                mixer = {"left": attention(L.mixer.left), "left_scale": L.mixer.left_scale,
                         "right": {"heads": r.heads, "vdim": r.vdim, "state": r.state, "groups": r.groups, "conv": r.taps,
                                   "norm_groups": r.norm_groups}, "right_scale": L.mixer.right_scale}
            mlp: Any = None
            if L.moe is not None:
                e = L.moe
                router: Dict[str, Any] = {"experts": e.experts, "top": e.top, "identity": e.identity, "scale": e.scale}
                if e.groups is not None:
                    router["groups"] = {"count": e.groups[0], "keep": e.groups[1]}
                mlp = {"kind": "moe", "router": router, "expert": {"ff": e.ff, "limit": e.limit}}
                if e.shared is not None:
                    mlp["shared"] = {"ff": e.shared[0], "limit": e.shared[1]}
            out["layers"].append({"type": L.type, "mixer": mixer, "mlp": mlp})
        return out


def _attention_part(W: int, a: Attention, prefix: str, out_bias: bool, value_mix: Optional[str]) -> dict:
    """Arguments of ``projected_spec`` for an attention mixer whose tensors begin with ``prefix``."""
    position = None
    if a.rot_base is not None and a.rot_dims:
        scaling = None if a.rot_scaling is None else dict(zip(("factor", "original", "fast", "slow"), a.rot_scaling))
        position = PartSpec("rope_yarn", {"rotary_dim": a.rot_dims, "theta": a.rot_base, "scaling": scaling,
                                          "neighbours": True})
    others = {"qkv.bias": tuple(f"{prefix}{n}.b" for n in ("q", "k", "v")), "sink": (f"{prefix}sink",)}
    if out_bias:
        others["o.bias"] = (f"{prefix}o.b",)
    if value_mix is not None:
        others["vmix"] = (f"{prefix}vmix",)
    return {"kind": "sink_attention",
            "args": {"hidden_size": W, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "key_dim": a.dim,
                     "value_dim": a.vdim, "scale": a.scale, "position": position, "window": a.window, "sink": True,
                     "gate": True, "qkv_bias": True, "out_bias": out_bias, "value_mix": value_mix},
            "segments": {"qkv": tuple(f"{prefix}{n}" for n in ("q", "k", "v")), "gate": (f"{prefix}g",)},
            "out": f"{prefix}o", "others": others}


def build_vudezen_spec(cfg: VudezenConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps
    norm = lambda name: PartSpec("layernorm", {"size": W, "eps": eps}, {"weight": (name,), "bias": (name + ".b",)})
    layers, mixed = [], False
    for i, L in enumerate(cfg.layers):
        p = f"l{i}"
        if L.type == "attention":
            value_mix = None
            if L.mixer.v_mix:            # the first such layer's values are what the others blend in
                value_mix, mixed = ("mixed" if mixed else "first"), True
            mixer = projected_spec(**_attention_part(W, L.mixer, f"{p}.mix.", True, value_mix))
        else:
            r, rp = L.mixer.right, f"{p}.mix.right."
            right = {"kind": "state_space",
                     "args": {"hidden_size": W, "num_heads": r.heads, "value_dim": r.vdim, "state_dim": r.state,
                              "groups": r.groups, "taps": r.taps, "norm_groups": r.norm_groups, "norm_eps": eps},
                     "segments": {"in": (rp + "in",)}, "out": rp + "o",
                     "others": {"conv.weight": (rp + "conv",), "conv.bias": (rp + "conv.b",), "dt_bias": (rp + "dt_bias",),
                                "A_log": (rp + "A_log",), "D": (rp + "D",), "norm": (rp + "norm",)}}
            mixer = summed_mixers_spec(W, {"left": _attention_part(W, L.mixer.left, f"{p}.mix.left.", False, None),
                                           "right": right},
                                       {"left": L.mixer.left_scale, "right": L.mixer.right_scale})
        parts = {"mixer_norm": norm(f"{p}.norm1"), "mixer": mixer, "mixer_post_norm": norm(f"{p}.norm1b")}
        if L.moe is not None:
            e = L.moe
            sources = {"router.weight": (f"{p}.mlp.router",), "correction": (f"{p}.mlp.correction",),
                       "gate_up.weight": tuple(f"{p}.mlp.e{j}.{n}" for j in range(e.experts) for n in ("gate", "up")),
                       "down.weight": tuple(f"{p}.mlp.e{j}.down" for j in range(e.experts))}
            if e.shared is not None:
                sources["shared.gate_up.weight"] = (f"{p}.mlp.shared.gate", f"{p}.mlp.shared.up")
                sources["shared.down.weight"] = (f"{p}.mlp.shared.down",)
            parts["ffn_norm"] = norm(f"{p}.norm2")
            parts["ffn"] = PartSpec(
                "routed_experts",
                {"hidden_size": W, "num_experts": e.experts, "top": e.top, "intermediate_size": e.ff,
                 "shared_size": e.shared[0] if e.shared else None, "score": "softmax", "renormalize": True,
                 "weight_on": "output", "correction": True, "groups": e.groups, "identity": e.identity,
                 "factor": e.scale, "sum_eps": _SUM_EPS, "limit": e.limit,
                 "shared_limit": e.shared[1] if e.shared else None},
                sources)
            parts["ffn_post_norm"] = norm(f"{p}.norm2b")
        layers.append(LayerSpec("sandwich", parts, {"residual_mult": cfg.residual_mult}))
    return ModelSpec(
        architecture=cfg.architecture,
        hidden_size=W,
        vocab_size=cfg.vocab,
        max_position=_MAX_POSITION,
        default_max_len=_DEFAULT_MAX_LEN,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": W}, {"weight": ("embed",)}),
        layers=tuple(layers),
        run_order=tuple(RunEntry(layer=i, cache=i) for i in range(len(layers))),
        final_norm=norm("final.norm"),
        lm_head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": W, "tied": False, "scale": cfg.logit_scale,
                                     "softcap": cfg.logit_softcap or 0.0}, {"weight": ("head",)}),
        # (a layer without a feed-forward has no use for the norms around one)
        ignored_tensors=tuple(rf"^l{i}\.norm2b?(\.b)?$" for i, L in enumerate(cfg.layers) if L.moe is None),
    )


register_architecture(VudezenConfig.ARCHITECTURE, VudezenConfig.from_dict, build_vudezen_spec)
