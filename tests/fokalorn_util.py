"""Small Fokalorn configurations and helpers shared by the Fokalorn tests."""
import json
import os

import torch

from dobelix_util import make_runner, sequences  # noqa: F401  (the same engine settings and token draws)


def dense(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def delta(heads, kv_heads, dim, vdim, conv, ff=None, ranks=None):
    """``ranks``: (decay, gate) rows of the low-rank projections; kept out of the config.json that is written."""
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": dense(ff), "_ranks": ranks or (6, 10)}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=1000.0, ff=None):
    return {"type": "latent_attention", "mlp": dense(ff),
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"base": base, "dims": rot_dim}}}


def config(width, vocab, layers, streams=3, groups=4, loop=None, eps=1e-5, scale=1.0):
    c = {"architecture": "Fokalorn", "vocab": vocab, "width": width, "streams": streams, "layers": layers,
         "norm": {"eps": eps, "groups": groups}, "embedding": {"scale": scale}}
    if loop is not None:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return c


# Two configurations that differ from each other in every size and option.  A: values wider than keys, shared query/key
# heads, a loop of three passes, three streams.  B: no loop, layers without feed-forward, one group, five streams (the
# kernel for any number), one tap, sizes of the tensor-core attention.
FOK_A = config(64, 200, [delta(4, 2, 16, 24, 4, ff=80), latent(4, 24, 8, 16, 40, 0.3, 500.0, ff=96), delta(3, 1, 32, 16, 2, ff=48),
                         latent(2, 16, 16, 40, 24, 0.25, 2.0e4, ff=72)], streams=3, groups=4, loop=(1, 3, 3), eps=1e-5, scale=3.0)
FOK_B = config(96, 310, [latent(5, 16, 32, 24, 64, 0.2, 77.0), delta(2, 2, 48, 40, 1, ff=64, ranks=(3, 17)),
                         latent(3, 8, 4, 8, 28, 0.4, 1.0e5, ff=56), delta(1, 1, 72, 88, 5)], streams=5, groups=1, eps=1e-6, scale=4.0)
STD = 0.15
MARK_A, MARK_B, MARK_LATER = 0, 1, 2      # embedding dimensions that mark the tokens of the far-token tests


def with_ranks(cfg):
    """The configuration with the ranks a checkpoint's tensors would tell."""
    cfg = json.loads(json.dumps(cfg))
    for layer in cfg["layers"]:
        ranks = layer.pop("_ranks", None)
        if layer["type"] == "channel_delta":
            layer["mixer"]["rank"], layer["mixer"]["gate_rank"] = ranks
    return cfg


def stored(cfg):
    """The configuration as config.json holds it."""
    cfg = json.loads(json.dumps(cfg))
    for layer in cfg["layers"]:
        layer.pop("_ranks", None)
    return cfg


def write_model(path, cfg, seed, dtype="bfloat16", edit=None):
    """A model folder with random weights (stored in ``dtype``); ``edit(tensors)`` may change them first.  Streams'
    coefficients, shifts, decays and sinks get values that spread over their useful ranges."""
    from hfee_b200.config.registry import resolve
    from hfee_b200.parts.model import model_tensor_needs
    from hfee_b200.weights.random_init import random_tensors
    from hfee_b200.weights.safetensors_io import write_file
    arch, typed = resolve(with_ranks(cfg))
    needs = model_tensor_needs(arch.build_spec(typed))
    tensors = random_tensors(needs, seed, torch.float32, STD)
    g = torch.Generator().manual_seed(seed)
    uniform = lambda t, lo, hi: t.copy_(torch.empty(t.shape).uniform_(lo, hi, generator=g))
    for name, t in sorted(tensors.items()):
        if name.endswith((".hc1.in", ".hc2.in")):
            uniform(t, 0.1, 0.9)
        elif name.endswith((".hc1.out", ".hc2.out")):
            uniform(t, 0.4, 1.4)
        elif name.endswith((".hc1.mix", ".hc2.mix")):
            uniform(t, -0.25, 0.25)
            t += torch.eye(t.shape[0])
        elif name.endswith(".shift"):
            uniform(t, 0.0, 0.9)
        elif name.endswith(".sink"):
            uniform(t, -1.0, 3.0)
        elif name.endswith(".A_log"):
            uniform(t, -3.0, 1.0)
        elif name.endswith(".dt_bias"):
            uniform(t, -4.0, 1.0)
        elif name.endswith((".a2", ".g2", ".mix.b")):
            t.mul_(3.0)                       # gates that move with the token
    if edit is not None:
        edit(tensors)
    store = {"bfloat16": torch.bfloat16, "float32": torch.float32}[dtype]
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(stored(cfg), f)
    write_file(os.path.join(path, "model.safetensors"), {k: v.to(store).contiguous() for k, v in tensors.items()})
    return path


def mark_first_tokens(tensors, size=1.0):
    """Tokens 0 and 1 (which the far-token tests put at chosen places only) carry a large entry in a dimension of their
    own and every other token in a third one, so that a projection can pick out "token A", "token B" and "any other
    token" by one column of its weight each."""
    emb = tensors["embed"]
    emb[:, [MARK_A, MARK_B, MARK_LATER]] = 0.0
    emb[0, MARK_A] = size
    emb[1, MARK_B] = size
    emb[2:, MARK_LATER] = size
