"""Designs whose layers are listed one by one in `config.json` (`architecture` names the design) and their checkpoints.

A design module gives `ARCHITECTURE`, `from_config` / `to_config` (config.json ⇄ `LayeredConfig`), `PRESETS`, and
`tensors(cfg)`: checkpoint tensor name → `Place`, where its values live in this package's (stacked) parameters.  Loading,
assembling and exporting checkpoints follow from that table.  A design whose config.json leaves sizes to the tensors' shapes says so
with `SIZES_FROM_TENSORS`: its `from_config` then also takes the checkpoint's shapes by name.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from functools import lru_cache

import torch

from .layered import LayeredConfig, layer_shapes


@dataclass(frozen=True)
class Place:
    """Part of a parameter: everything, or [start, stop) of leading dimensions (one pair per dimension; a single entry of the first
    dimension is (e, e + 1) with `squeeze`)."""

    param: str
    at: tuple = ()
    squeeze: bool = False

    def of(self, t: torch.Tensor) -> torch.Tensor:
        v = t[tuple(slice(a, b) for a, b in self.at)] if self.at else t
        return v.squeeze(0) if self.squeeze else v


def design(cfg):
    """The module of a configuration's design, None for the other families."""
    return DESIGNS.get(getattr(cfg, "family", None))


@lru_cache(maxsize=8)
def table(cfg: LayeredConfig) -> dict[str, Place]:
    return design(cfg).tensors(cfg)


def param_shapes(cfg: LayeredConfig) -> dict[str, tuple]:
    H, V = cfg.hidden_size, cfg.vocab_size
    out = {"embed": (V, H), "norm": (H,)}
    if not cfg.tie_embeddings:
        out["lm_head"] = (V, H)
    if cfg.bigram is not None:
        out["bigram"] = (cfg.bigram.buckets + 1, H)
    if cfg.token_side:
        out["side_embed"] = (V, cfg.num_layers * cfg.token_side)
    for i, s in enumerate(cfg.layer_specs):
        out.update({f"layers.{i}.{n}": shape for n, shape in layer_shapes(s, cfg).items()})
    return out


def is_checkpoint(names, cfg: LayeredConfig) -> bool:
    """Names of the design's files (not this package's own)."""
    t = table(cfg)
    return any(n in t and t[n].param != n for n in names)


def load_into(params: dict, named, cfg: LayeredConfig) -> set:
    """Copy checkpoint tensors (any subset: the parts of a stack may come apart) into the model's parameters.  Returns the
    parameters of which every value was given."""
    given: dict[str, int] = {}
    for name, t in named:
        where = table(cfg).get(name)
        if where is None:
            continue
        dst = where.of(params[where.param].data)
        assert tuple(t.shape) == tuple(dst.shape), f"{name}: got {tuple(t.shape)}, the configuration says {tuple(dst.shape)}"
        dst.copy_(t)
        given[where.param] = given.get(where.param, 0) + dst.numel()
    return {n for n, k in given.items() if k >= params[n].numel()}


def from_checkpoint(named: dict[str, torch.Tensor], cfg: LayeredConfig) -> dict[str, torch.Tensor]:
    """Full parameters of this package from a checkpoint's tensors (those of which every part is there)."""
    shapes, out, given = param_shapes(cfg), {}, {}
    for name, where in table(cfg).items():
        if name not in named:
            continue
        t = named[name]
        if not where.at:
            assert tuple(t.shape) == shapes[where.param], f"{name}: got {tuple(t.shape)}, the configuration says {shapes[where.param]}"
            out[where.param] = t
            continue
        if where.param not in given:
            out[where.param], given[where.param] = torch.empty(shapes[where.param], dtype=t.dtype, device=t.device), 0
        dst = where.of(out[where.param])
        assert tuple(t.shape) == tuple(dst.shape), f"{name}: got {tuple(t.shape)}, the configuration says {tuple(dst.shape)}"
        dst.copy_(t)
        given[where.param] += t.numel()
    return {n: t for n, t in out.items() if given.get(n, math.prod(shapes[n])) == math.prod(shapes[n])}


def to_checkpoint(name: str, tensor: torch.Tensor, cfg: LayeredConfig) -> list[tuple[str, torch.Tensor]]:
    """One parameter of this package → the checkpoint's tensors."""
    return [(n, where.of(tensor)) for n, where in table(cfg).items() if where.param == name]


def rows_of(param: str, parts) -> dict[str, Place]:
    """Places of tensors stacked along the rows: `parts` = (name, rows)."""
    out, at = {}, 0
    for n, rows in parts:
        out[n] = Place(param, ((at, at + rows),))
        at += rows
    return out


from . import nopelorn, ronupel, senadra, vozirax  # noqa: E402  (they use Place and rows_of)

DESIGNS = {"nopelorn": nopelorn, "ronupel": ronupel, "vozirax": vozirax, "senadra": senadra}
