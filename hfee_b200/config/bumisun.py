"""Typed configuration of the Bumisun decoder, read from its config.json.

A Bumisun model norms its embedding, runs a list of pre-norm layers whose sublayers' outputs are all scaled by
``residual_mult``, and scales its logits.  Each layer has one of two mixers (``attention``: grouped-query softmax attention
with a partial rotation, capped scores, a window behind which the first tokens stay visible, a sink, and values mixed with
the first mixing layer's; ``mamba2``: a state-space scan with one decay per head behind a short convolution, a gate in
front of a norm in parts) and an optional feed-forward (``dense``: relu-gated; ``moe``: routed experts weighted by a softmax
over the chosen logits, with an optional gated shared expert).  Every size and every constant that differs between models
comes from config.json; nothing here has a default that a model could silently fall back on.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .dobelix import DenseMlp, _get, _int, _num
from .llama import ConfigError
from .muvetar import Expert, _expert
from .pupinex import _count, _positive


@dataclass(frozen=True)
class BumisunAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float]
    window: Optional[int]
    keep_first: int
    rot_dims: int            # 0: no rotation
    rot_base: float
    v_mix: bool


@dataclass(frozen=True)
class Mamba2Mixer:
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_groups: int


@dataclass(frozen=True)
class ChosenMoe:
    experts: int
    top: int
    expert: Expert
    shared: Optional[Expert]


@dataclass(frozen=True)
class BumisunLayer:
    type: str
    mixer: Any
    mlp: Any                 # DenseMlp, ChosenMoe or None


@dataclass(frozen=True)
class BumisunConfig:
    vocab: int
    width: int
    layers: Tuple[BumisunLayer, ...]
    eps: float
    residual_mult: float
    logit_scale: float
    max_positions: int

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "BumisunConfig":
        layers = _get(d, "layers", "config")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        out = []
        for i, entry in enumerate(layers):
            where = f"layers[{i}]"
            kind = _get(entry, "type", where)
            m = _get(entry, "mixer", where)
            mw = where + ".mixer"
            if kind == "attention":
                mixer = _attention(m, mw)
            elif kind == "mamba2":
                mixer = _mamba2(m, mw)
            else:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of this design (known: attention, mamba2)")
            out.append(BumisunLayer(kind, mixer, _mlp(entry.get("mlp"), where + ".mlp")))
        mixing = [l.mixer for l in out if l.type == "attention" and l.mixer.v_mix]
        for m in mixing[1:]:
            if (m.kv_heads, m.vdim) != (mixing[0].kv_heads, mixing[0].vdim):
                raise ConfigError("config.json: layers that mix values must have values of one size, got "
                                  f"{m.kv_heads} x {m.vdim} beside {mixing[0].kv_heads} x {mixing[0].vdim}")
        max_positions = d.get("max_positions", d.get("max_position_embeddings", 1 << 20))
        return cls(vocab=_int(d, "vocab", "config"), width=_int(d, "width", "config"), layers=tuple(out),
                   eps=_num(_get(d, "norm", "config"), "eps", "norm"), residual_mult=_num(d, "residual_mult", "config"),
                   logit_scale=_num(d, "logit_scale", "config"), max_positions=int(max_positions))


def _attention(m: Mapping[str, Any], where: str) -> BumisunAttention:
    heads, kv = _int(m, "heads", where), _int(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"config.json: {where}.heads {heads} must be a multiple of kv_heads {kv}")
    dim = _int(m, "dim", where)
    rot, dims, base = m.get("rot"), 0, 1.0
    if rot is not None:
        dims = _count(rot, "dims", where + ".rot")
        if dims % 2 or dims > dim:
            raise ConfigError(f"config.json: {where}.rot.dims {dims} must be even and at most dim {dim}")
        base = _positive(rot, "base", where + ".rot") if dims else 1.0
    mask, window, keep = m.get("mask"), None, 0
    if mask is not None:                     # no mask: every earlier position
        window, keep = _int(mask, "size", where + ".mask"), _count(mask, "keep_first", where + ".mask")
    cap = None if m.get("softcap") is None else _positive(m, "softcap", where)
    v_mix = m.get("v_mix", False)
    if not isinstance(v_mix, bool):
        raise ConfigError(f"config.json: {where}.v_mix must be true or false, got {v_mix!r}")
    return BumisunAttention(heads, kv, dim, _int(m, "vdim", where), _num(m, "scale", where), cap, window, keep, dims, base, v_mix)


def _mamba2(m: Mapping[str, Any], where: str) -> Mamba2Mixer:
    heads, vdim, groups, parts = (_int(m, k, where) for k in ("heads", "vdim", "groups", "norm_groups"))
    if heads % groups:
        raise ConfigError(f"config.json: {where}.heads {heads} must be a multiple of groups {groups}")
    if (heads * vdim) % parts:
        raise ConfigError(f"config.json: {where}.norm_groups {parts} does not divide the {heads * vdim} columns of heads x vdim")
    return Mamba2Mixer(heads, vdim, _int(m, "state", where), groups, _int(m, "conv", where), parts)


def _mlp(mlp: Optional[Mapping[str, Any]], where: str):
    if mlp is None:
        return None
    kind = _get(mlp, "kind", where)
    if kind == "dense":
        return DenseMlp(_int(mlp, "ff", where))
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind {kind!r} is not a feed-forward of this design (known: dense, moe)")
    router = _get(mlp, "router", where)
    experts, top = _int(router, "experts", where + ".router"), _int(router, "top", where + ".router")
    if top > experts:
        raise ConfigError(f"config.json: {where}.router.top {top} exceeds its {experts} experts")
    shared = mlp.get("shared")
    return ChosenMoe(experts, top, _expert(_get(mlp, "expert", where), where + ".expert"),
                     None if shared is None else _expert(shared, where + ".shared"))
