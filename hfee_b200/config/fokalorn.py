"""Typed configuration of the Fokalorn decoder, read from its config.json.

A Fokalorn model keeps several residual streams beside one another (``streams``) that every sublayer reads as a weighted
sum and writes back through a small matrix, norms in groups (``norm.groups``), mixes each mixer's input with the row of
the token before, and may run a stretch of its layers several times over with the same weights (``loop``).  Each layer
has one of two mixers (``channel_delta``: a gated delta rule whose state decays per key channel, behind short
convolutions; ``latent_attention``: softmax attention over one cached latent and one shared rotated key part per token,
with a sink and a gate per head) and an optional ``dense`` feed-forward.  Every size and every constant that differs
between models comes from config.json or a tensor's shape; nothing here has a default that a model could silently fall
back on.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .dobelix import DenseMlp, _get, _int, _num
from .llama import ConfigError
from .pupinex import Loop, _count, _positive


@dataclass(frozen=True)
class ChannelDeltaMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    decay_rank: int          # rows of the decay's and of the output gate's low-rank projections (from the tensors' shapes)
    gate_rank: int


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float


@dataclass(frozen=True)
class FokalornLayer:
    type: str
    mixer: Any
    mlp: Optional[DenseMlp]


@dataclass(frozen=True)
class FokalornConfig:
    vocab: int
    width: int
    streams: int
    layers: Tuple[FokalornLayer, ...]
    loop: Optional[Loop]
    eps: float
    groups: int
    embedding_scale: float
    max_positions: int

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "FokalornConfig":
        layers = _get(d, "layers", "config")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        out = []
        for i, entry in enumerate(layers):
            where = f"layers[{i}]"
            kind = _get(entry, "type", where)
            m = _get(entry, "mixer", where)
            mw = where + ".mixer"
            if kind == "channel_delta":
                heads, kv = _int(m, "heads", mw), _int(m, "kv_heads", mw)
                if heads % kv:
                    raise ConfigError(f"config.json: {mw}.heads {heads} must be a multiple of kv_heads {kv}")
                for key, tensor in (("rank", "a1"), ("gate_rank", "g1")):
                    if not isinstance(m, Mapping) or m.get(key) is None:
                        raise ConfigError(f"config.json: {mw}: {key} is neither given nor known from the tensor l{i}.mix.{tensor}")
                mixer = ChannelDeltaMixer(heads, kv, _int(m, "dim", mw), _int(m, "vdim", mw),
                                          _int(m, "conv", mw), int(m["rank"]), int(m["gate_rank"]))
            elif kind == "latent_attention":
                rot_dim = _int(m, "rot_dim", mw)
                rot = _get(m, "rot", mw)
                dims = _int(rot, "dims", mw + ".rot")
                if dims != rot_dim or dims % 2:
                    raise ConfigError(f"config.json: {mw}.rot.dims {dims} must be even and equal rot_dim {rot_dim}: the whole "
                                      "shared key part is rotated")
                mixer = LatentMixer(_int(m, "heads", mw), _int(m, "dim", mw), rot_dim, _int(m, "vdim", mw),
                                    _int(m, "kv_rank", mw), _num(m, "scale", mw), _positive(rot, "base", mw + ".rot"))
            else:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of this design (known: channel_delta, latent_attention)")
            mlp = entry.get("mlp") if isinstance(entry, Mapping) else None
            if mlp is not None:
                mk = _get(mlp, "kind", where + ".mlp")
                if mk != "dense":
                    raise ConfigError(f"config.json: {where}.mlp.kind {mk!r} is not a feed-forward of this design (known: dense)")
                mlp = DenseMlp(_int(mlp, "ff", where + ".mlp"))
            out.append(FokalornLayer(kind, mixer, mlp))
        loop = d.get("loop")
        if loop is not None:
            loop = Loop(_count(loop, "start", "loop"), _count(loop, "stop", "loop"), _int(loop, "times", "loop"))
            if not (0 <= loop.start <= loop.stop <= len(out)) or loop.times < 1:
                raise ConfigError(f"config.json: loop {loop.start}..{loop.stop} x {loop.times} does not fit {len(out)} layers")
        norm = _get(d, "norm", "config")
        width, groups = _int(d, "width", "config"), _int(norm, "groups", "norm")
        if width % groups:
            raise ConfigError(f"config.json: norm.groups {groups} does not divide the width {width}")
        max_positions = d.get("max_positions", d.get("max_position_embeddings", 1 << 20))
        return cls(vocab=_int(d, "vocab", "config"), width=width, streams=_int(d, "streams", "config"),
                   layers=tuple(out), loop=loop, eps=_num(norm, "eps", "norm"), groups=groups,
                   embedding_scale=_num(_get(d, "embedding", "config"), "scale", "embedding"), max_positions=int(max_positions))


def fill_from_tensors(config_json: Mapping[str, Any], shapes: Mapping[str, Tuple[int, ...]]) -> Mapping[str, Any]:
    """config.json does not name the ranks of a ``channel_delta`` layer's low-rank projections: they are the row counts
    of its ``mix.a1`` (decay) and ``mix.g1`` (output gate) tensors."""
    layers = config_json.get("layers")
    if not isinstance(layers, (list, tuple)):
        return config_json
    new_layers = []
    for i, entry in enumerate(layers):
        if isinstance(entry, Mapping) and entry.get("type") == "channel_delta" and isinstance(entry.get("mixer"), Mapping):
            found = {key: int(shapes[f"l{i}.mix.{tensor}"][0]) for key, tensor in (("rank", "a1"), ("gate_rank", "g1"))
                     if f"l{i}.mix.{tensor}" in shapes}
            entry = dict(entry, mixer={**entry["mixer"], **found})
        new_layers.append(entry)
    return dict(config_json, layers=new_layers)
