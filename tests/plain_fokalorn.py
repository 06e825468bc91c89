"""Plain, slow Fokalorn decoder used as the oracle of the test-suite.

Whole sequences only, no cache, no batching, one function per mechanism, numpy float64 throughout, loops over
tokens where the definition is a recurrence.  It shares no code with the ``hfee_b200`` package: its own safetensors
reader and its own reading of config.json.

The design, in the notation used below (X: the residual streams [streams, T, width]; N: RMS norm in groups):

    X_1 = .. = X_s = table[token] * scale
    sublayer q of a layer run:   u = sum_s a[s] X_s;   y = f(N(u));   X_t <- sum_s M[s, t] X_s + b[t] y
    (f: the mixer on token-shifted rows first, then the feed-forward if the layer has one)
    a stretch of layers runs several times over with the same weights
    logits = head . N(sum_s X_s)

Two mixers: ``channel_delta`` (a gated delta rule whose state decays per key channel, behind short convolutions) and
``latent_attention`` (softmax attention over one cached latent and one shared rotated key part per token, with a sink
and a gate per head).  One feed-forward: squared relu between two products.
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


def group_norm(x, w, eps, groups):
    """RMS norm of every one of ``groups`` equal consecutive parts of a row, then a weight per column."""
    parts = x.reshape(x.shape[:-1] + (groups, x.shape[-1] // groups))
    return unit_rms(parts, eps).reshape(x.shape) * w


def token_shift(h, mu):
    """h_t + (h_(t-1) - h_t) * mu with h_(-1) = 0."""
    before = np.concatenate([np.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def collect_streams(X, a):
    """What a sublayer sees of the streams."""
    return np.tensordot(a, X, axes=(0, 0))


def spread_streams(X, M, b, y):
    """The streams after a sublayer that returned y: M is indexed [from, to]."""
    out = np.zeros_like(X)
    for t in range(X.shape[0]):
        out[t] = b[t] * y
        for s in range(X.shape[0]):
            out[t] += M[s, t] * X[s]
    return out


def short_conv(x, w):
    """y[t, c] = sum_j w[c, j] x[t - taps + 1 + j, c], zeros in front of the sequence."""
    T, taps = x.shape[0], w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    return sum(padded[j:j + T] * w[:, j] for j in range(taps))


def unit_vectors(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def channel_delta_scan(q, k, v, beta, g):
    """q, k [T, H, d] (a head's own copies), v [T, H, dv], beta [T, H], g [T, H, d] -> o [T, H, dv]."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2]))
    out = np.zeros_like(v)
    for t in range(T):
        S = S * g[t][:, :, None]
        u = beta[t][:, None] * (v[t] - np.einsum("hdc,hd->hc", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hdc,hd->hc", S, q[t])
    return out


def channel_delta(m, w, p, h, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in "qkv")
    q = unit_vectors(q.reshape(T, G, d)) * d ** -0.5
    k = unit_vectors(k.reshape(T, G, d))
    share = np.arange(H) // (H // G)
    beta = sigmoid(h @ w[p + "b"].T)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    g = np.exp(-np.exp(w[p + "A_log"])[None, :, None] * softplus(z).reshape(T, H, d))
    o = channel_delta_scan(q[:, share], k[:, share], v.reshape(T, H, dv), beta, g)
    gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
    return ((unit_rms(o, eps) * w[p + "norm"]).reshape(T, H * dv) * gate) @ w[p + "o"].T


def rotate(x, dims, base):
    """x [T, heads, r]: the pair (2i, 2i + 1) of a row at position p turns by p * base^(-2i/dims)."""
    a = np.arange(x.shape[0])[:, None] * np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.copy()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def sink_softmax(scores, sink):
    """Rows of scores (-inf: not seen); the denominator has one more term exp(sink)."""
    top = np.maximum(scores.max(axis=-1), sink)
    e = np.exp(scores - top[:, None])
    return e / (e.sum(axis=-1) + np.exp(sink - top))[:, None]


def latent_attention(m, w, p, h, eps):
    T = h.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).reshape(T, H, d + r)
    down = h @ w[p + "dkv"].T
    c = unit_rms(down[:, :rank], eps) * w[p + "dkv.norm"]
    k = (c @ w[p + "uk"].T).reshape(T, H, d)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    dims, base = m["rot"]["dims"], m["rot"]["base"]
    q_rot = rotate(q[..., d:], dims, base)
    k_rot = rotate(down[:, None, rank:], dims, base)[:, 0]
    seen = np.tril(np.ones((T, T), dtype=bool))
    gate = sigmoid(h @ w[p + "g"].T)
    out = np.zeros((T, H, dv))
    for i in range(H):
        s = (q[:, i, :d] @ k[:, i].T + q_rot[:, i] @ k_rot.T) * m["scale"]
        weights = sink_softmax(np.where(seen, s, -np.inf), w[p + "sink"][i])
        out[:, i] = weights @ v[:, i] * gate[:, i:i + 1]
    return out.reshape(T, H * dv) @ w[p + "o"].T


def squared_relu_mlp(w, p, h):
    return np.maximum(h @ w[p + "up"].T, 0.0) ** 2 @ w[p + "down"].T


MIXERS = {"channel_delta": channel_delta, "latent_attention": latent_attention}


# --------------------------------------------------------------------------
# the model
# --------------------------------------------------------------------------
def run_order(cfg):
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return list(range(n))
    lo, hi = loop["start"], loop["stop"]
    return list(range(lo)) + list(range(lo, hi)) * loop["times"] + list(range(hi, n))


def layer(cfg, w, i, X):
    """The streams after layer i."""
    spec, p = cfg["layers"][i], f"l{i}."
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    h = group_norm(collect_streams(X, w[p + "hc1.in"]), w[p + "norm1"], eps, groups)
    h = token_shift(h, w[p + "shift"])
    y = MIXERS[spec["type"]](spec["mixer"], w, p + "mix.", h, eps)
    X = spread_streams(X, w[p + "hc1.mix"], w[p + "hc1.out"], y)
    if spec.get("mlp"):
        h = group_norm(collect_streams(X, w[p + "hc2.in"]), w[p + "norm2"], eps, groups)
        X = spread_streams(X, w[p + "hc2.mix"], w[p + "hc2.out"], squared_relu_mlp(w, p + "mlp.", h))
    return X


def forward(cfg, w, tokens, residuals=None):
    """Logits [T, vocab]; ``residuals`` (a list) takes the sum of the streams after every layer run."""
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    X = np.repeat(x[None], cfg["streams"], axis=0)
    for i in run_order(cfg):
        X = layer(cfg, w, i, X)
        if residuals is not None:
            residuals.append(X.sum(axis=0))
    x = group_norm(X.sum(axis=0), w["final.norm"], cfg["norm"]["eps"], cfg["norm"]["groups"])
    return x @ w["head"].T


def greedy(cfg, w, prompt, count):
    toks = list(prompt)
    for _ in range(count):
        toks.append(int(np.argmax(forward(cfg, w, toks)[-1])))
    return toks[len(prompt):]
