"""The Bumisun decoder as an arrangement of parts.

    x = N_embed(table[token])
    a layer:   x += r * mixer(N_1(x));   x += r * ffn(N_2(x))        (the second only if the layer has a feed-forward)
    logits = logit_scale * head(N_final(x))

N: RMS norm, r: ``residual_mult``.  Layer i's tensors are named ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*`` and
``l<i>.mlp.*``; model level: ``embed``, ``embed.norm``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.bumisun import BumisunConfig
from ..config.dobelix import DenseMlp
from ..config.registry import register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec

SWISH_ALPHA = 1.702          # fixed by the design: g * sigmoid(1.702 g) (u + 1) in the experts


def _mixer(cfg: BumisunConfig, layer, p: str, value_mix):
    m = layer.mixer
    if layer.type == "attention":
        position = (PartSpec("rotary", head_dim=m.dim, rope_dim=m.rot_dims, theta=m.rot_base, scaling=None, pairing="half")
                    if m.rot_dims > 0 else PartSpec("none"))
        spec = PartSpec("softmax_attention", width=cfg.width, heads=m.heads, kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim,
                        scale=m.scale, softcap=m.softcap, window=m.window, keep_first=m.keep_first, position=position, sink=True,
                        value_mix=value_mix)
        keys = ("q", "k", "v", "o", "sink") + (("vmix",) if value_mix is not None else ())
        return spec, {"mixer." + k: p + "mix." + k for k in keys}
    spec = PartSpec("head_scan", width=cfg.width, heads=m.heads, head_dim=m.vdim, state=m.state, groups=m.groups, taps=m.taps,
                    norm_parts=m.norm_groups, eps=cfg.eps)
    stored = {"conv_bias": "conv.b"}
    return spec, {"mixer." + k: p + "mix." + stored.get(k, k)
                  for k in ("in", "conv", "conv_bias", "dt_bias", "A_log", "D", "norm", "o")}


def _feed_forward(cfg: BumisunConfig, f, p: str):
    if isinstance(f, DenseMlp):
        return (PartSpec("gated", width=cfg.width, inner=f.ff, activation="relu"),
                {"ffn." + k: p + "mlp." + k for k in ("gate", "up", "down")})
    shared = f.shared
    spec = PartSpec("routed_experts", width=cfg.width, experts=f.experts, top=f.top, router_scale=1.0, inner=f.expert.ff,
                    limit=f.expert.limit, alpha=SWISH_ALPHA, shift=1.0, router="softmax_chosen", router_bias=True,
                    shared_inner=None if shared is None else shared.ff, shared_limit=None if shared is None else shared.limit,
                    shared_gate=shared is not None)
    names = {"ffn.router": p + "mlp.router", "ffn.router.b": p + "mlp.router.b"}
    for e in range(f.experts):
        for k in ("gate", "up", "down"):
            names[f"ffn.e{e}.{k}"] = f"{p}mlp.e{e}.{k}"
    if shared is not None:
        for k in ("gate", "up", "down", "sg"):
            names[f"ffn.shared.{k}"] = f"{p}mlp.shared.{k}"
    return spec, names


def bumisun_spec(cfg: BumisunConfig) -> ModelSpec:
    norm = PartSpec("rms_norm", width=cfg.width, eps=cfg.eps)
    block = PartSpec("scaled_pre_norm", width=cfg.width, residual_scale=cfg.residual_mult)
    layers, ignorable = [], []
    mixing = False           # whether an earlier layer has left its values for the ones that mix
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        value_mix = None
        if layer.type == "attention" and layer.mixer.v_mix:
            value_mix, mixing = ("mixed" if mixing else "first"), True
        elif layer.type == "attention":       # a file may carry the unused share of a layer that does not mix
            ignorable.append(p + "mix.vmix")
        mixer, names = _mixer(cfg, layer, p, value_mix)
        names["mixer_norm.weight"] = p + "norm1"
        parts = {"mixer": ("mixer", mixer), "mixer_norm": ("norm", norm)}
        if layer.mlp is not None:
            ffn, ffn_names = _feed_forward(cfg, layer.mlp, p)
            parts.update(ffn=("feed_forward", ffn), ffn_norm=("norm", norm))
            names.update(ffn_names)
            names["ffn_norm.weight"] = p + "norm2"
        else:                                 # likewise the unused norm of a layer without feed-forward
            ignorable.append(p + "norm2")
        layers.append(LayerSpec(block, parts, names))
    return ModelSpec(
        width=cfg.width, vocab=cfg.vocab,
        embedding=PartSpec("token", vocab=cfg.vocab, width=cfg.width, norm_eps=cfg.eps),
        layers=tuple(layers), schedule=ModelSpec.sequential(len(layers)), final_norm=norm,
        head=PartSpec("linear", vocab=cfg.vocab, width=cfg.width, tied=False, scale=cfg.logit_scale),
        names={"embedding.table": "embed", "embedding.norm": "embed.norm", "final_norm.weight": "final.norm", "head.weight": "head"},
        max_positions=cfg.max_positions, ignorable=tuple(ignorable))


register_architecture("Bumisun", BumisunConfig.from_dict, bumisun_spec)
