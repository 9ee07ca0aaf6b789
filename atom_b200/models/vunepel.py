"""Vunepel: a decoder-only model whose layers are listed one by one in config.json.  Every layer has one norm (a dynamic
tanh, without mean or variance) whose output both its sub-blocks read, and adds both outputs to the residual stream.  The
mixer is a gated delta rule with a decay per key channel, or differential attention within chunks of positions, whose keys
and values may be another such layer's; the feed-forward is dense with clamped gates, a mixture of experts of that form
beside a gated shared one, or absent.

config.json:  ``architecture`` "Vunepel"; ``vocab``, ``width``; ``norm.eps``;
``layers``: entries with ``type`` ("channel_delta" | "attention"), ``mixer``, ``mlp`` (or null)
  channel_delta mixer: heads, kv_heads, dim, vdim, conv (taps); the ranks of the decay's and the output gate's projections
      stand in the checkpoint's shapes (without a checkpoint: keys decay_rank and gate_rank)
  attention mixer: heads, kv_heads, dim (per map), vdim, scale, diff, rot {base, dims} (absent: no rotation), mask {size}
      (absent: every earlier token is seen), kv_from (absent: keys and values of its own)
  mlp: {kind "dense", ff, limit} or {kind "moe", router {experts, top, scale}, expert {ff, limit}, shared {ff, limit}
      (absent: none)}

Tensors: ``embed``, ``head``, ``final.norm``, per layer ``l<i>.norm1`` (every norm with ``<name>.b`` and a number
``<name>.alpha``) and
  channel_delta: ``l<i>.mix.{q,k,v}`` with ``.conv`` each, ``l<i>.mix.{b,A_log,a1,a2,dt_bias,g1,g2,norm,o}``
  attention:     ``l<i>.mix.{q,q.norm,lq1,lk1,lq2,lk2,o}``, without kv_from also ``l<i>.mix.{k,k.norm,v}``
  dense:         ``l<i>.mlp.{gate,up,down}``
  moe:           ``l<i>.mlp.router``, ``l<i>.mlp.e<j>.{gate,up,down}``, ``l<i>.mlp.shared.{gate,up,down,sg}``
Matrices are [out, in].

  x = embed[token]
  per layer:  h = tanh(alpha x) * w + b;   x += mixer(h) + mlp(h)
  logits = head (tanh(alpha x) * w + b)
The mixers' formulas stand in parts/delta_rule.py and parts/differential_attention.py, the feed-forwards' in parts/mlp.py
(gated_clamped) and parts/moe.py (routed_experts).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, ClassVar, Dict, List, Mapping, Optional, Tuple

from ..config.model_config import ConfigError, ModelConfig, cfg_get, cfg_positive
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunEntry
from ..parts.summed_mixers import projected_spec
from .registry import register_architecture

# Nothing in the design bounds a position (angles are computed from the position itself); a request's length is
# bounded by the engine's max_model_len, which defaults to this many tokens.
_DEFAULT_MAX_LEN = 32768
_MAX_POSITION = 1 << 24        # positions are exact in 32-bit floats up to here

_SUM_EPS = 1e-20               # added to the sum that the chosen experts' scores are divided by


@dataclass(frozen=True)
class Delta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    decay_rank: int
    gate_rank: int


@dataclass(frozen=True)
class Attention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    rot_base: Optional[float]
    rot_dims: int
    chunk: Optional[int]
    kv_from: Optional[int]


@dataclass(frozen=True)
class Dense:
    ff: int
    limit: float


@dataclass(frozen=True)
class Experts:
    experts: int
    top: int
    scale: float
    ff: int
    limit: float
    shared: Optional[Dense]


@dataclass(frozen=True)
class VunepelLayer:
    type: str
    mixer: Any                       # Delta | Attention
    mlp: Any                         # Dense | Experts | None


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


def _heads(m: Mapping, w: str) -> Tuple[int, int, int, int]:
    h, g = _count(m, "heads", w), _count(m, "kv_heads", w)
    if h % g:
        raise ConfigError(f"config.json: {w}heads ({h}) must be a multiple of kv_heads ({g})")
    return h, g, _count(m, "dim", w), _count(m, "vdim", w)


def _delta(m: Mapping, w: str, prefix: str, shapes) -> Delta:
    def rank(tensor: str, key: str) -> int:
        if shapes is None:
            return _count(m, key, w)          # (without a checkpoint the ranks are keys)
        shape = shapes.get(prefix + tensor)
        if shape is None or len(shape) != 2:
            raise ConfigError(f"checkpoint: no matrix '{prefix}{tensor}', whose rows give a rank")
        return int(shape[0])

    h, g, d, dv = _heads(m, w)
    return Delta(h, g, d, dv, _count(m, "conv", w), rank("a1", "decay_rank"), rank("g1", "gate_rank"))


def _attention(m: Mapping, w: str) -> Attention:
    base, dims, chunk, kv_from = None, 0, None, None
    h, g, d, dv = _heads(m, w)
    if m.get("rot") is not None:
        rot = _obj(m, "rot", w)
        base, dims = _positive(rot, "base", w + "rot."), _count(rot, "dims", w + "rot.", 0)
        if dims % 2 or dims > d:
            raise ConfigError(f"config.json: {w}rot.dims ({dims}) must be even and at most dim ({d})")
    if m.get("mask") is not None:
        chunk = _count(_obj(m, "mask", w), "size", w + "mask.")
    if m.get("kv_from") is not None:
        kv_from = _count(m, "kv_from", w, 0)
    return Attention(h, g, d, dv, _number(m, "scale", w), _number(m, "diff", w), base, dims, chunk, kv_from)


def _mlp(mlp, w: str):
    if mlp is None:
        return None
    kind = mlp.get("kind") if isinstance(mlp, dict) else mlp
    dense = lambda d, where: Dense(_count(d, "ff", where), _positive(d, "limit", where))
    if kind == "dense":
        return dense(mlp, w + "mlp.")
    if kind != "moe":
        raise ConfigError(f"config.json: {w}mlp must be null or an object of kind 'dense' or 'moe', got {kind!r}")
    w += "mlp."
    r, e = _obj(mlp, "router", w), dense(_obj(mlp, "expert", w), w + "expert.")
    shared = dense(_obj(mlp, "shared", w), w + "shared.") if mlp.get("shared") is not None else None
    out = Experts(_count(r, "experts", w + "router."), _count(r, "top", w + "router."),
                  _number(r, "scale", w + "router.") if r.get("scale") is not None else 1.0, e.ff, e.limit, shared)
    if out.top > out.experts:
        raise ConfigError(f"config.json: {w}router.top ({out.top}) exceeds the number of experts ({out.experts})")
    return out


@dataclass(frozen=True)
class VunepelConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm_eps: float = 0.0
    layers: Tuple[VunepelLayer, ...] = ()

    ARCHITECTURE: ClassVar[str] = "Vunepel"

    @classmethod
    def from_dict(cls, d: Dict[str, Any], shapes: Optional[Mapping[str, Tuple[int, ...]]] = None) -> "VunepelConfig":
        """shapes: checkpoint tensor name -> shape, when the configuration is read beside a checkpoint."""
        entries = d.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers: List[VunepelLayer] = []
        for i, e in enumerate(entries):
            w = f"layers[{i}]."
            if not isinstance(e, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = e.get("type")
            m = _obj(e, "mixer", w)
            if kind == "attention":
                mixer: Any = _attention(m, w + "mixer.")
                if mixer.kv_from is not None:
                    j = mixer.kv_from
                    owner = layers[j] if j < i else None
                    if owner is None or owner.type != "attention" or owner.mixer.kv_from is not None:
                        raise ConfigError(f"config.json: {w}mixer.kv_from ({j}) must be an earlier attention layer with "
                                          "keys and values of its own")
                    o = owner.mixer
                    if (o.kv_heads, o.dim, o.vdim) != (mixer.kv_heads, mixer.dim, mixer.vdim):
                        raise ConfigError(f"config.json: {w}mixer: the keys and values of layer {j} have other sizes")
            elif kind == "channel_delta":
                mixer = _delta(m, w + "mixer.", f"l{i}.mix.", shapes)
            else:
                raise ConfigError(f"config.json: {w}type {kind!r} is not supported (channel_delta, attention)")
            layers.append(VunepelLayer(kind, mixer, _mlp(e.get("mlp"), w)))
        return cls(architecture=cls.ARCHITECTURE, vocab=cfg_positive("vocab", cfg_get(d, "vocab", int)),
                   width=cfg_positive("width", cfg_get(d, "width", int)),
                   norm_eps=_positive(_obj(d, "norm", ""), "eps", "norm."), layers=tuple(layers))

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                               "norm": {"eps": self.norm_eps}, "layers": []}
        for L in self.layers:
            a = L.mixer
            m: Dict[str, Any] = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim}
            if L.type == "channel_delta":
                m.update(conv=a.taps, decay_rank=a.decay_rank, gate_rank=a.gate_rank)
            else:
                m.update(scale=a.scale, diff=a.diff)
                if a.rot_base is not None:
                    m["rot"] = {"base": a.rot_base, "dims": a.rot_dims}
                if a.chunk is not None:
                    m["mask"] = {"size": a.chunk}
                if a.kv_from is not None:
                    m["kv_from"] = a.kv_from
            mlp: Any = None
            if isinstance(L.mlp, Dense):
                mlp = {"kind": "dense", "ff": L.mlp.ff, "limit": L.mlp.limit}
            elif L.mlp is not None:
                e = L.mlp
                mlp = {"kind": "moe", "router": {"experts": e.experts, "top": e.top, "scale": e.scale},
                       "expert": {"ff": e.ff, "limit": e.limit}}
                if e.shared is not None:
                    mlp["shared"] = {"ff": e.shared.ff, "limit": e.shared.limit}
            out["layers"].append({"type": L.type, "mixer": m, "mlp": mlp})
        return out


def _held(chunks: List[Optional[int]]) -> Optional[Tuple[int, bool]]:
    """How far back readers of one cache with these chunks look: (window, whether it is a chunk), None for everything.
    Chunks of different sizes lie within a sliding window of the largest."""
    if any(c is None for c in chunks):
        return None
    return max(chunks), len(set(chunks)) == 1


def _ffn(W: int, mlp, p: str) -> PartSpec:
    if isinstance(mlp, Dense):
        return PartSpec("gated_clamped", {"hidden_size": W, "intermediate_size": mlp.ff, "limit": mlp.limit},
                        {"gate_up.weight": (f"{p}gate", f"{p}up"), "down.weight": (f"{p}down",)})
    e = mlp
    sources = {"router.weight": (f"{p}router",),
               "gate_up.weight": tuple(f"{p}e{j}.{n}" for j in range(e.experts) for n in ("gate", "up")),
               "down.weight": tuple(f"{p}e{j}.down" for j in range(e.experts))}
    if e.shared is not None:      # (the shared expert's gate is one more row of the router's product)
        sources["router.weight"] += (f"{p}shared.sg",)
        sources["shared.gate_up.weight"] = (f"{p}shared.gate", f"{p}shared.up")
        sources["shared.down.weight"] = (f"{p}shared.down",)
    return PartSpec("routed_experts",
                    {"hidden_size": W, "num_experts": e.experts, "top": e.top, "intermediate_size": e.ff,
                     "shared_size": e.shared.ff if e.shared else None, "score": "sigmoid", "renormalize": True,
                     "weight_on": "output", "shared_gate": e.shared is not None, "factor": e.scale, "sum_eps": _SUM_EPS,
                     "limit": e.limit, "shared_limit": e.shared.limit if e.shared else None}, sources)


def build_vunepel_spec(cfg: VunepelConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps
    norm = lambda n: PartSpec("dynamic_tanh", {"size": W}, {"weight": (n,), "bias": (n + ".b",), "alpha": (n + ".alpha",)})
    readers: Dict[int, List[Optional[int]]] = {}
    for i, L in enumerate(cfg.layers):
        if L.type == "attention":
            readers.setdefault(i if L.mixer.kv_from is None else L.mixer.kv_from, []).append(L.mixer.chunk)
    layers, order = [], []
    for i, L in enumerate(cfg.layers):
        p, a, owner = f"l{i}.mix.", L.mixer, i
        if L.type == "attention":
            own = a.kv_from is None
            owner = i if own else a.kv_from
            position = None
            if a.rot_base is not None and a.rot_dims:
                position = PartSpec("rope_yarn", {"rotary_dim": a.rot_dims, "theta": a.rot_base})
            others = {"lambdas": tuple(p + n for n in ("lq1", "lk1", "lq2", "lk2")), "q_norm": (p + "q.norm",)}
            if own:
                others["k_norm"] = (p + "k.norm",)
            mixer = projected_spec(
                "differential_attention",
                {"hidden_size": W, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "key_dim": a.dim, "value_dim": a.vdim,
                 "scale": a.scale, "diff": a.diff, "norm_eps": eps, "position": position, "chunk": a.chunk,
                 "own_keys": own, "held": _held(readers[owner])},
                {"qkv": tuple(p + n for n in (("q", "k", "v") if own else ("q",)))}, p + "o", others)
        else:
            mixer = projected_spec(
                "channel_delta_rule",
                {"hidden_size": W, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "key_dim": a.dim, "value_dim": a.vdim,
                 "taps": a.taps, "decay_rank": a.decay_rank, "gate_rank": a.gate_rank, "norm_eps": eps},
                {"qkv": (p + "q", p + "k", p + "v"), "a": (p + "a1",), "g": (p + "g1",), "b": (p + "b",)}, p + "o",
                {"conv.weight": tuple(f"{p}{n}.conv" for n in ("q", "k", "v")), "a2.weight": (p + "a2",),
                 "g2.weight": (p + "g2",), "A_log": (p + "A_log",), "dt_bias": (p + "dt_bias",), "norm": (p + "norm",)})
        parts = {"norm": norm(f"l{i}.norm1"), "mixer": mixer}
        if L.mlp is not None:
            parts["ffn"] = _ffn(W, L.mlp, f"l{i}.mlp.")
        layers.append(LayerSpec("parallel", parts))
        order.append(RunEntry(layer=i, cache=owner, writes_cache=owner == i))
    return ModelSpec(
        architecture=cfg.architecture,
        hidden_size=W,
        vocab_size=cfg.vocab,
        max_position=_MAX_POSITION,
        default_max_len=_DEFAULT_MAX_LEN,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": W}, {"weight": ("embed",)}),
        layers=tuple(layers),
        run_order=tuple(order),
        final_norm=norm("final.norm"),
        lm_head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": W, "tied": False}, {"weight": ("head",)}),
    )


register_architecture(VunepelConfig.ARCHITECTURE, VunepelConfig.from_dict, build_vunepel_spec, reads_shapes=True)
