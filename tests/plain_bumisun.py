"""Plain, slow Bumisun decoder used as the oracle of the test-suite.

Whole sequences only, no cache, no batching, one function per mechanism, numpy float64 throughout, loops over
tokens where the definition is a recurrence.  It shares no code with the ``hfee_b200`` package: its own safetensors
reader and its own reading of config.json.

The design, in the notation used below (x: the residual stream [T, width]; N: RMS norm with a weight; r: the residual
multiplier):

    x = N_embed(table[token])
    a layer:   x <- x + r mixer(N_1(x));   x <- x + r ffn(N_2(x))     (the second only if the layer has a feed-forward)
    logits = (head . N_final(x)) * logit_scale

Two mixers: ``attention`` (grouped-query attention with a partial rotation, capped scores, a window that keeps the
first tokens in sight, a sink, and values mixed with the first mixing layer's) and ``mamba2`` (a state-space recurrence
with one decay per head behind a short convolution, a gate in front of a norm in parts).  Two feed-forwards: a gated one
with relu, and routed experts with clamped gates beside a gated shared expert.
"""
from __future__ import annotations

import json
import os
import struct

import numpy as np


def read_safetensors(path):
    """name -> float64 (or integer) ndarray; bfloat16 is widened by a 16-bit shift."""
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        blob = f.read()
    kinds = {"F64": "<f8", "F32": "<f4", "F16": "<f2", "I32": "<i4", "I64": "<i8"}
    out = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        lo, hi = meta["data_offsets"]
        raw = blob[lo:hi]
        if meta["dtype"] == "BF16":
            u = np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16
            arr = u.view(np.float32).astype(np.float64)
        else:
            arr = np.frombuffer(raw, dtype=kinds[meta["dtype"]])
            if arr.dtype.kind == "f":
                arr = arr.astype(np.float64)
        out[name] = arr.reshape(meta["shape"])
    return out


def load(model_dir):
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(model_dir, "model.safetensors"))


# --------------------------------------------------------------------------
# one function per mechanism
# --------------------------------------------------------------------------
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def unit_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def norm_in_parts(x, w, eps, parts):
    """RMS norm of every one of ``parts`` equal consecutive parts of a row, then a weight per column."""
    pieces = x.reshape(x.shape[:-1] + (parts, x.shape[-1] // parts))
    return unit_rms(pieces, eps).reshape(x.shape) * w


def rotate(x, dims, base):
    """x [T, heads, d]: of the leading ``dims`` dimensions the pair (i, i + dims/2) of a row at position p turns by
    p * base^(-2i/dims)."""
    half = dims // 2
    a = np.arange(x.shape[0])[:, None] * np.array([base ** (-2.0 * i / dims) for i in range(half)])[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def cap(score, limit):
    return score if limit is None else limit * np.tanh(score / limit)


def visible(T, size, keep_first):
    """[query, key]: not in the future, and inside the window or among the kept first tokens."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    seen = j <= i
    return seen if size is None else seen & ((i - j < size) | (j < keep_first))


def sink_softmax(scores, sink):
    """Rows of scores (-inf: not seen); the denominator has one more term exp(sink)."""
    top = np.maximum(scores.max(axis=-1), sink)
    e = np.exp(scores - top[:, None])
    return e / (e.sum(axis=-1) + np.exp(sink - top))[:, None]


def mix_values(v, first, share):
    return (1.0 - share) * v + share * first


def attention(m, w, p, h, eps, memo):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, d)
    k = (h @ w[p + "k"].T).reshape(T, G, d)
    v = (h @ w[p + "v"].T).reshape(T, G, dv)
    rot = m.get("rot")
    if rot:
        q, k = rotate(q, rot["dims"], rot["base"]), rotate(k, rot["dims"], rot["base"])
    if m.get("v_mix"):
        if "first_values" in memo:
            v = mix_values(v, memo["first_values"], float(w[p + "vmix"]))
        else:
            memo["first_values"] = v
    mask = m.get("mask") or {}
    seen = visible(T, mask.get("size"), mask.get("keep_first", 0))
    out = np.zeros((T, H, dv))
    for i in range(H):
        g = i // (H // G)
        s = cap((q[:, i] @ k[:, g].T) * m["scale"], m.get("softcap"))
        out[:, i] = sink_softmax(np.where(seen, s, -np.inf), w[p + "sink"][i]) @ v[:, g]
    return out.reshape(T, H * dv) @ w[p + "o"].T


def short_conv(x, w, b):
    """y[t, c] = b[c] + sum_j w[c, j] x[t - taps + 1 + j, c], zeros in front of the sequence."""
    T, taps = x.shape[0], w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    return b + sum(padded[j:j + T] * w[:, j] for j in range(taps))


def head_scan(x, B, C, dt, A, D):
    """x [T, H, dv], B, C [T, H, N] (a head's own copies), dt [T, H], A, D [H] -> y [T, H, dv]."""
    T, H, dv = x.shape
    S = np.zeros((H, B.shape[2], dv))
    out = np.zeros_like(x)
    for t in range(T):
        S = np.exp(-A * dt[t])[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        out[t] = np.einsum("hnc,hn->hc", S, C[t]) + D[:, None] * x[t]
    return out


def mamba2(m, w, p, h, eps, memo):
    T = h.shape[0]
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    proj = h @ w[p + "in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    xbc = silu(short_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    share = np.arange(H) // (H // G)
    x = xbc[:, :inner].reshape(T, H, dv)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)[:, share]
    C = xbc[:, inner + G * N:].reshape(T, G, N)[:, share]
    y = head_scan(x, B, C, softplus(dt + w[p + "dt_bias"]), np.exp(w[p + "A_log"]), w[p + "D"])
    y = norm_in_parts(y.reshape(T, inner) * silu(z), w[p + "norm"], eps, m["norm_groups"])
    return y @ w[p + "o"].T


def relu_gated_mlp(w, p, h):
    return (np.maximum(h @ w[p + "gate"].T, 0.0) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def clamped_expert(w, p, h, limit):
    g = np.minimum(h @ w[p + "gate"].T, limit)
    u = np.clip(h @ w[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


ROUTE_MARGINS = []       # per call: the smallest gap between a chosen logit and the best one left out


def choose(logits, top):
    """(experts [T, top], weights [T, top]): the largest logits and the softmax over just those."""
    chosen = np.argsort(-logits, axis=-1, kind="stable")[:, :top]
    if top < logits.shape[-1]:
        ranked = np.sort(logits, axis=-1)[:, ::-1]
        ROUTE_MARGINS.append(float((ranked[:, top - 1] - ranked[:, top]).min()))
    e = np.take_along_axis(logits, chosen, axis=-1)
    e = np.exp(e - e.max(axis=-1, keepdims=True))
    return chosen, e / e.sum(axis=-1, keepdims=True)


def routed_experts(f, w, p, h):
    chosen, weight = choose(h @ w[p + "router"].T + w[p + "router.b"], f["router"]["top"])
    out = np.zeros_like(h)
    for e in range(f["router"]["experts"]):
        t, slot = np.nonzero(chosen == e)
        if len(t):
            out[t] += weight[t, slot][:, None] * clamped_expert(w, f"{p}e{e}.", h[t], f["expert"]["limit"])
    if f.get("shared"):
        out += clamped_expert(w, p + "shared.", h, f["shared"]["limit"]) * sigmoid(h @ w[p + "shared.sg"].T)
    return out


MIXERS = {"attention": attention, "mamba2": mamba2}


# --------------------------------------------------------------------------
# the model
# --------------------------------------------------------------------------
def layer(cfg, w, i, x, memo):
    spec, p = cfg["layers"][i], f"l{i}."
    eps, r = cfg["norm"]["eps"], cfg["residual_mult"]
    x = x + r * MIXERS[spec["type"]](spec["mixer"], w, p + "mix.", rms_norm(x, w[p + "norm1"], eps), eps, memo)
    mlp = spec.get("mlp")
    if mlp:
        h = rms_norm(x, w[p + "norm2"], eps)
        x = x + r * (relu_gated_mlp(w, p + "mlp.", h) if mlp["kind"] == "dense" else routed_experts(mlp, w, p + "mlp.", h))
    return x


def forward(cfg, w, tokens, residuals=None):
    """Logits [T, vocab]; ``residuals`` (a list) takes the stream after every layer."""
    x = rms_norm(w["embed"][np.asarray(tokens)], w["embed.norm"], cfg["norm"]["eps"])
    memo = {}
    for i in range(len(cfg["layers"])):
        x = layer(cfg, w, i, x, memo)
        if residuals is not None:
            residuals.append(x)
    return (rms_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T) * cfg["logit_scale"]


def greedy(cfg, w, prompt, count):
    toks = list(prompt)
    for _ in range(count):
        toks.append(int(np.argmax(forward(cfg, w, toks)[-1])))
    return toks[len(prompt):]
