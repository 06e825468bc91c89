"""Small Bumisun configurations and helpers shared by the Bumisun tests."""
import json
import os

import torch

from dobelix_util import make_runner, sequences  # noqa: F401  (the same engine settings and token draws)


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, shared_ff=None, shared_limit=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if shared_ff is not None:
        m["shared"] = {"ff": shared_ff, "limit": shared_limit}
    return m


def attn(heads, kv_heads, dim, vdim, size=None, keep=0, rot=0, base=1000.0, scale=0.3, softcap=None, v_mix=False, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if size is not None:
        m["mask"] = {"size": size, "keep_first": keep}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
    if softcap is not None:
        m["softcap"] = softcap
    return {"type": "attention", "mixer": m, "mlp": mlp}


def mamba(heads, vdim, state, groups, conv, norm_groups, mlp=None):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                                   "norm_groups": norm_groups}}


def config(width, vocab, layers, eps=1e-5, residual_mult=0.6, logit_scale=1.7):
    return {"architecture": "Bumisun", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "residual_mult": residual_mult, "logit_scale": logit_scale}


# Two configurations that differ from each other in every size and option.  A: the first layer mixes values, windows that keep
# first tokens, groups of scan heads, norms in parts.  B: a scan first, the first mixing layer is the third, attention without
# window, without rotation or without cap, one tap, a layer without feed-forward, one chosen expert, no shared one.
BUM_A = config(64, 200, [attn(4, 2, 16, 24, 21, 5, rot=8, scale=0.3, softcap=4.0, v_mix=True, mlp=dense(80)),
                         mamba(4, 24, 16, 2, 3, 2, mlp=moe(6, 2, 24, 0.9, 40, 1.1)),
                         attn(6, 2, 32, 24, 13, 2, rot=32, base=50.0, scale=0.2, softcap=2.0, v_mix=True, mlp=moe(5, 3, 16, 1.5)),
                         attn(2, 1, 24, 40, 34, 17, rot=16, base=2.0e4, scale=0.4, softcap=9.0),
                         mamba(3, 16, 40, 1, 4, 3, mlp=dense(56)),
                         attn(4, 2, 8, 24, 50, 1, rot=4, base=300.0, scale=0.5, softcap=6.0, v_mix=True, mlp=dense(48))],
               eps=1e-5, residual_mult=0.6, logit_scale=1.7)
BUM_B = config(96, 310, [mamba(5, 16, 24, 5, 1, 1),
                         attn(3, 3, 40, 16, scale=0.25, mlp=moe(12, 1, 8, 2.0, 24, 0.7)),
                         attn(8, 1, 16, 32, 40, 0, rot=16, base=77.0, scale=0.35, softcap=3.0, v_mix=True, mlp=dense(72)),
                         mamba(2, 72, 8, 1, 5, 2, mlp=moe(3, 3, 32, 5.0, 8, 0.4)),
                         attn(2, 1, 16, 32, 5, 40, rot=2, base=9.0, scale=0.3, v_mix=True),
                         mamba(8, 16, 64, 4, 2, 2, mlp=moe(4, 2, 40, 0.8))],
               eps=1e-6, residual_mult=1.0, logit_scale=0.5)
STD = 0.15
LOUD_EMBEDDING = 3.0                      # the embedding's random entries are this many times larger (its norm levels rows anyway)
MARK_A, MARK_B, MARK_LATER = 0, 1, 2      # embedding dimensions that mark the tokens of the far-token tests
ROUTE_AT = 3                              # first of the embedding dimensions that name a token's experts


def clear_routes(tensors, cfg, loud=3.0):
    """Make every router's choice a clear call, so that rounding cannot flip one.  Every layer with experts gets embedding
    dimensions of its own, one per expert, which its router reads with weight 3 (and everything else with a tenth of its
    random weight); token t is loud in the dimensions of the ``top`` experts from t % experts on (cyclically), and no sublayer's
    output projection writes into those dimensions.  Mixers and earlier layers still move the scores, so the chosen experts'
    weights differ from token to token."""
    emb = tensors["embed"]
    at = ROUTE_AT
    for i, layer in enumerate(cfg["layers"]):
        if (layer.get("mlp") or {}).get("kind") != "moe":
            continue
        experts, top = layer["mlp"]["router"]["experts"], layer["mlp"]["router"]["top"]
        assert at + experts <= emb.shape[1], "the width has no room for every layer's marks"
        w = tensors[f"l{i}.mlp.router"]
        w.mul_(0.1)
        emb[:, at:at + experts] = 0.0
        for e in range(experts):
            w[e, at:at + experts] = 0.0
            w[e, at + e] = 3.0
        for t in range(emb.shape[0]):
            for k in range(top):
                emb[t, at + (t + k) % experts] = loud
        at += experts
    for name, t in tensors.items():          # no sublayer writes into the marks: they reach every router as the embedding left them
        if name.endswith((".o", ".down")):
            t[ROUTE_AT:at] = 0.0


def write_model(path, cfg, seed, dtype="bfloat16", edit=None, routes=True):
    """A model folder with random weights (stored in ``dtype``); ``edit(tensors)`` may change them first.  Decays, step sizes,
    sinks and shares get values that spread over their useful ranges."""
    from hfee_b200.config.registry import resolve
    from hfee_b200.parts.model import model_tensor_needs
    from hfee_b200.weights.random_init import random_tensors
    from hfee_b200.weights.safetensors_io import write_file
    arch, typed = resolve(cfg)
    needs = model_tensor_needs(arch.build_spec(typed))
    tensors = random_tensors(needs, seed, torch.float32, STD)
    tensors["embed"].mul_(LOUD_EMBEDDING)
    g = torch.Generator().manual_seed(seed)
    uniform = lambda t, lo, hi: t.copy_(torch.empty(t.shape).uniform_(lo, hi, generator=g))
    for name, t in sorted(tensors.items()):
        if name.endswith(".sink"):
            uniform(t, -1.0, 3.0)
        elif name.endswith(".vmix"):
            uniform(t, 0.2, 0.9)
        elif name.endswith(".A_log"):
            uniform(t, -3.0, 1.0)
        elif name.endswith(".dt_bias"):
            uniform(t, -3.0, 1.0)
        elif name.endswith(".mix.D"):
            uniform(t, 0.5, 1.5)
        elif name.endswith((".conv", ".conv.b")):
            t.mul_(3.0)
        elif name.endswith(".router.b"):
            uniform(t, -0.3, 0.3)
    if routes and any((l.get("mlp") or {}).get("kind") == "moe" for l in cfg["layers"]):
        clear_routes(tensors, cfg)
    if edit is not None:
        edit(tensors)
    store = {"bfloat16": torch.bfloat16, "float32": torch.float32}[dtype]
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_file(os.path.join(path, "model.safetensors"), {k: v.to(store).contiguous() for k, v in tensors.items()})
    return path


def mark_tokens(tensors, size=1.0):
    """Tokens 0 and 1 (which the tests put at chosen places only) carry a large entry in a dimension of their own and every
    other token in a third one, so that a projection can pick out "token A", "token B" and "any other token" by one column of
    its weight each."""
    emb = tensors["embed"]
    emb[:, [MARK_A, MARK_B, MARK_LATER]] = 0.0
    emb[0, MARK_A] = size
    emb[1, MARK_B] = size
    emb[2:, MARK_LATER] = size


def smallest_route_margin(plain, cfg, weights, seqs):
    """The smallest gap, over all routed tokens and layers, between a chosen expert's logit and the best one left out."""
    del plain.ROUTE_MARGINS[:]
    for s in seqs:
        plain.forward(cfg, weights, s)
    return min(plain.ROUTE_MARGINS) if plain.ROUTE_MARGINS else float("inf")
