"""The Fokalorn decoder as an arrangement of parts.

    X_1 = .. = X_s = table[token] * scale
    sublayer q of a layer run:   u = sum_s a_q[s] X_s;   y = f(N_q(u));   X_t <- sum_s M_q[s, t] X_s + b_q[t] y
    q = 1: the mixer, which reads h_t + (h_(t-1) - h_t) * mu of the normed rows h;  q = 2: the feed-forward, if any
    layers loop.start .. loop.stop - 1 run loop.times times in a row with the same weights, a cache of its own per pass
    logits = head . N(sum_s X_s)

N: RMS norm in groups.  Layer i's tensors are named ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.shift``, ``l<i>.hc1.*``,
``l<i>.hc2.*``, ``l<i>.mix.*`` and ``l<i>.mlp.*``; model level: ``embed``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.fokalorn import FokalornConfig, fill_from_tensors
from ..config.registry import register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec


def _mixer(cfg: FokalornConfig, layer, p: str):
    m = layer.mixer
    if layer.type == "latent_attention":
        position = PartSpec("rotary", head_dim=m.rot_dim, rope_dim=m.rot_dim, theta=m.rot_base, scaling=None, pairing="interleaved")
        spec = PartSpec("latent_attention", width=cfg.width, heads=m.heads, head_dim=m.dim, rope_dim=m.rot_dim, value_dim=m.vdim,
                        q_rank=None, kv_rank=m.kv_rank, position=position, scale=m.scale, window=None, eps=cfg.eps, gate="head",
                        sink=True)
        keys = ("q", "dkv", "dkv_norm", "uk", "uv", "sink", "g", "o")
    else:
        spec = PartSpec("channel_delta_rule", width=cfg.width, heads=m.heads, qk_heads=m.kv_heads, key_dim=m.dim, value_dim=m.vdim,
                        taps=m.taps, decay_rank=m.decay_rank, gate_rank=m.gate_rank, eps=cfg.eps)
        keys = ("q", "k", "v", "q_conv", "k_conv", "v_conv", "b", "a1", "a2", "A_log", "dt_bias", "norm", "g1", "g2", "o")
    stored = {"dkv_norm": "dkv.norm", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv"}
    return spec, {f"mixer.{k}": p + "mix." + stored.get(k, k) for k in keys}


def fokalorn_spec(cfg: FokalornConfig) -> ModelSpec:
    norm = PartSpec("group_rms_norm", width=cfg.width, eps=cfg.eps, groups=cfg.groups)
    streams = PartSpec("hyper_connection", streams=cfg.streams)
    block = PartSpec("hyper_connected", width=cfg.width)
    layers, ignorable = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        mixer, names = _mixer(cfg, layer, p)
        names.update({"mixer_norm.weight": p + "norm1", "mixer_shift.weight": p + "shift",
                      **{f"mixer_streams.{k}": f"{p}hc1.{k}" for k in ("in", "out", "mix")}})
        parts = {"mixer": ("mixer", mixer), "mixer_norm": ("norm", norm), "mixer_streams": ("streams", streams),
                 "mixer_shift": ("shift", PartSpec("token_shift", width=cfg.width))}
        if layer.mlp is not None:
            parts.update(ffn=("feed_forward", PartSpec("dense", width=cfg.width, inner=layer.mlp.ff, activation="relu2")),
                         ffn_norm=("norm", norm), ffn_streams=("streams", streams))
            names.update({"ffn.up": p + "mlp.up", "ffn.down": p + "mlp.down", "ffn_norm.weight": p + "norm2",
                          **{f"ffn_streams.{k}": f"{p}hc2.{k}" for k in ("in", "out", "mix")}})
        else:           # a file may carry the unused norm and coefficients of a layer without feed-forward
            ignorable += [p + "norm2", p + "hc2.*"]
        layers.append(LayerSpec(block, parts, names))
    loop = cfg.loop
    schedule = (ModelSpec.sequential(len(layers)) if loop is None else
                ModelSpec.looped(len(layers), loop.start, loop.stop, loop.times))
    return ModelSpec(
        width=cfg.width, vocab=cfg.vocab,
        embedding=PartSpec("token", vocab=cfg.vocab, width=cfg.width, scale=cfg.embedding_scale),
        layers=tuple(layers), schedule=schedule, final_norm=norm,
        head=PartSpec("linear", vocab=cfg.vocab, width=cfg.width, tied=False),
        names={"embedding.table": "embed", "final_norm.weight": "final.norm", "head.weight": "head"},
        max_positions=cfg.max_positions, streams=cfg.streams, ignorable=tuple(ignorable))


register_architecture("Fokalorn", FokalornConfig.from_dict, fokalorn_spec, fill_from_tensors)
