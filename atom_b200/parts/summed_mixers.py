"""Two or more mixers side by side on the same input, their outputs added with a factor each:
   y = sum_m scale_m * mixer_m(x).

The members are mixers of the form W_o f(W_in x) (``ProjectedMixer``), so they share their products: all W_in are one
stacked matrix, each f takes its columns of the one projection and writes its rows, times its factor (in 32-bit, before
the rows are rounded), side by side into one array, and all W_o lie side by side in one matrix,
   y = [scale_1 f_1 | scale_2 f_2 | ...] [W_o,1 | W_o,2 | ...]^T.
Parameters of the members beside their products appear under ``<member>.<name>``; what the members keep between steps is
put together into one need (``CacheNeed.merged``) and each sees its own share of the run entry's cache slot.
"""
from __future__ import annotations

from typing import Dict, Mapping

import torch

from . import registry
from .base import ProjectedMixer
from .linear import linear
from .registry import register
from .spec import CacheNeed, ParamSpec, PartSpec


def projected_spec(kind: str, args: Mapping, segments: Mapping[str, tuple], out, others: Mapping[str, tuple]) -> PartSpec:
    """PartSpec of a ``ProjectedMixer``: segments: segment -> checkpoint tensors stacked in it (in whatever order the part
    lays the segments out); out: the output matrix's tensor; others: parameter -> checkpoint tensors."""
    part = registry.build("mixer", PartSpec(kind, dict(args)))
    names, _, _ = part.layout(part.segments())
    return PartSpec(kind, dict(args), {"in.weight": tuple(t for n in names for t in segments[n]), "o.weight": (out,), **others})


def summed_mixers_spec(hidden_size: int, members: Mapping[str, dict], scales: Mapping[str, float]) -> PartSpec:
    """members: name -> keyword arguments of ``projected_spec``."""
    args = {"hidden_size": hidden_size, "members": {n: PartSpec(m["kind"], dict(m["args"])) for n, m in members.items()},
            "scales": dict(scales)}
    segments = {f"{n}.{k}": v for n, m in members.items() for k, v in m["segments"].items()}
    others = {f"{n}.{k}": v for n, m in members.items() for k, v in m["others"].items()}
    spec = projected_spec("summed_mixers", args, segments, None, others)
    spec.sources["o.weight"] = tuple(m["out"] for m in members.values())
    return spec


@register("mixer", "summed_mixers")
class SummedMixers(ProjectedMixer):
    def __init__(self, hidden_size: int, members: Mapping[str, PartSpec], scales: Mapping[str, float]):
        self.hidden_size = hidden_size
        self.members = {n: registry.build("mixer", m) for n, m in members.items()}
        self.scales = {n: float(scales[n]) for n in members}
        for n, m in self.members.items():
            if not isinstance(m, ProjectedMixer) or m.hidden_size != hidden_size or m.out_bias:
                raise ValueError(f"summed_mixers: member '{n}' cannot share its products")
        self.inner_cols = sum(m.inner_cols for m in self.members.values())

    @property
    def graph_safe(self) -> bool:
        return all(m.graph_safe for m in self.members.values())

    def segments(self):
        return {f"{n}.{k}": v for n, m in self.members.items() for k, v in m.segments().items()}

    def params(self) -> Dict[str, ParamSpec]:
        cols = tuple(m.inner_cols for m in self.members.values())
        p = {"in.weight": self._in_spec(),
             "o.weight": ParamSpec((self.hidden_size, sum(cols)), rows=cols, stack_dim=1)}
        for n, m in self.members.items():
            p.update({f"{n}.{k}": v for k, v in m.inner_params().items()})
        return p

    def cache_need(self):
        return CacheNeed.merged({n: m.cache_need() for n, m in self.members.items()})

    def bind(self, tensors, rt):
        super().bind({k: tensors[k] for k in ("in.weight", "o.weight")}, rt)
        for n, m in self.members.items():
            m.bind({k[len(n) + 1:]: v for k, v in tensors.items() if k.startswith(n + ".")}, rt)

    def after_load(self) -> None:
        for m in self.members.values():
            m.after_load()

    def launch_plan(self, step) -> None:
        for m in self.members.values():
            m.launch_plan(step)

    def inner(self, x, proj, step, cache, writes_cache, y, y_scale):
        at = 0
        own_of = {n: {} for n in self.members}
        for k, v in proj.items():
            n, _, segment = k.partition(".")
            own_of[n][segment] = v
        for n, m in self.members.items():
            own = own_of[n]
            m.inner(x, own, step, cache.member(n), writes_cache, y[:, at:at + m.inner_cols], y_scale * self.scales[n])
            at += m.inner_cols
