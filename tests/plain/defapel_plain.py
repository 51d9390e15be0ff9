"""A plain, slow Defapel forward pass: one whole sequence from position 0, no cache, one function per mechanism.

It shares no code with ``purhie_b200``: it reads ``config.json`` with ``json`` and the weight file by its byte
layout, and states every equation directly.  Everything runs in float64.

The design in short (names of config.json in quotes):

* x <- x + mixer(norm1(x)); x <- x + experts(norm2(x)) where the layer has an "mlp".  norm(x) = rms(x) (1 + w).
* Mixer "channel_delta": per head a matrix S [dim, vdim] that first decays by a factor per key channel and is then
  corrected towards v along k:  S <- g S, S <- S + k (beta (v - S^T k))^T, o = S^T q.  q, k and v pass a short causal
  convolution and silu; q and k are unit vectors; g = exp(-exp(A_log) softplus(W_a2 W_a1 h + dt_bias)); o is RMS-normed per
  head and multiplied by sigmoid(W_g2 W_g1 h).
* Mixer "parallel": "left_scale" left(h) + "right_scale" right(h).  Left: grouped attention over the last "mask.size"
  positions, biases on q, k and v, q and k RMS-normed over all their heads at once, rotation of neighbouring pairs with
  stretched frequencies, scores through "softcap", heads gated by sigmoid(W_g h).  Right: the delta rule with one decay per
  head and a silu gate from one matrix.
* Experts: the "top" ones by sigmoid(W_router h); each runs on its score times h; the outputs are added.
* logits = "logit_scale" embed norm(x).
"""
import json
import os
import struct

import numpy as np


# ---- files ---------------------------------------------------------------------------------------------------------
def read_safetensors(path):
    """{name: float64 array (int tables stay int)}: 8-byte little-endian header length, the JSON header (name ->
    dtype, shape, data_offsets), the data."""
    with open(path, "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        header = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        lo, hi = meta["data_offsets"]
        raw = data[lo:hi]
        kind = meta["dtype"]
        if kind == "BF16":
            a = (np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        elif kind == "F32":
            a = np.frombuffer(raw, dtype="<f4").astype(np.float64)
        elif kind == "I32":
            a = np.frombuffer(raw, dtype="<i4").copy()
        else:
            raise ValueError(f"{name}: dtype {kind}")
        out[name] = a.reshape(meta["shape"])
    return out


def read_model(folder):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(folder, "model.safetensors"))


# ---- small functions -----------------------------------------------------------------------------------------------
def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.maximum(x, 0.0) + np.log1p(np.exp(-np.abs(x)))


def rms(x, eps, w=1.0):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


# ---- the delta rule ------------------------------------------------------------------------------------------------
def causal_conv(x, taps):
    """x [n, channels]: y_i = sum_j taps[:, j] x_(i - K + 1 + j), zeros before the start."""
    K = taps.shape[1]
    pad = np.concatenate([np.zeros((K - 1, x.shape[1])), x])
    return sum(taps[:, j] * pad[j:j + x.shape[0]] for j in range(K))


def delta_scan(q, k, v, beta, g, S=None):
    """q and k [n, H, D], v [n, H, V], beta [n, H], g [n, H, D] -> o [n, H, V] and the last S [H, D, V], token by token."""
    n, H, D = q.shape
    S = np.zeros((H, D, v.shape[2])) if S is None else S.copy()
    o = np.empty(v.shape)
    for t in range(n):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    return o, S


def delta_decay(z, a_log, bias):
    """z [n, H, D] (D may be 1) -> exp(-exp(A_log_h) softplus(z + bias))."""
    return np.exp(-np.exp(a_log)[:, None] * softplus(z + bias))


def delta_inputs(h, w, p, m):
    """q, k [n, H, D] and v [n, H, V] as they enter the recurrence."""
    n = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + c].T, w[p + c + ".conv"])) for c in "qkv")
    of = np.arange(H) // (H // G)
    q = unit(q.reshape(n, G, D))[:, of] * D ** -0.5
    k = unit(k.reshape(n, G, D))[:, of]
    return q, k, v.reshape(n, H, V)


def channel_delta(h, w, p, m, eps):
    n, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = delta_inputs(h, w, p, m)
    beta = sigmoid(h @ w[p + "b"].T)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T
    g = delta_decay(z.reshape(n, H, D), w[p + "A_log"], w[p + "dt_bias"].reshape(H, D))
    o, _ = delta_scan(q, k, v, beta, g)
    gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
    return (rms(o, eps, w[p + "norm"]).reshape(n, H * V) * gate) @ w[p + "o"].T


def head_delta(h, w, p, m, eps):
    n, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = delta_inputs(h, w, p, m)
    beta = sigmoid(h @ w[p + "b"].T)
    g = delta_decay((h @ w[p + "a"].T)[:, :, None], w[p + "A_log"], w[p + "dt_bias"][:, None])
    o, _ = delta_scan(q, k, v, beta, np.broadcast_to(g, (n, H, D)))
    return (rms(o, eps, w[p + "norm"]).reshape(n, H * V) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- attention -----------------------------------------------------------------------------------------------------
def frequencies(rot):
    """Per pair: base^(-2 i / dims), stretched by "factor" where the wavelength is long for "original" positions."""
    f = rot["base"] ** (-2.0 * np.arange(rot["dims"] // 2) / rot["dims"])
    s = rot.get("scaling")
    if not s:
        return f
    out = []
    for fi in f:
        wave = 2.0 * np.pi / fi
        if wave < s["original"] / s["high"]:
            out.append(fi)
        elif wave > s["original"] / s["low"]:
            out.append(fi / s["factor"])
        else:
            t = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
            out.append((1.0 - t) * fi / s["factor"] + t * fi)
    return np.array(out)


def rotate(x, rot, first=0):
    """x [n, heads, dim], row 0 at position ``first``: the first "dims" of each head in pairs (2i, 2i + 1)."""
    y = x.copy()
    dims = rot["dims"]
    a = (first + np.arange(x.shape[0]))[:, None, None] * frequencies(rot)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    y[..., 0:dims:2] = u * np.cos(a) - v * np.sin(a)
    y[..., 1:dims:2] = v * np.cos(a) + u * np.sin(a)
    return y


def window_seen(n, size):
    d = np.arange(n)[:, None] - np.arange(n)[None, :]
    return (d >= 0) & (d < size)


def softmax_rows(s, seen):
    s = np.where(seen, s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def window_attention(h, w, p, m, eps):
    n = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[p + c].T + w[p + c + ".b"] for c in "qkv")
    q = rotate(rms(q, eps, w[p + "q.norm"]).reshape(n, H, D), m["rot"])
    k = rotate(rms(k, eps, w[p + "k.norm"]).reshape(n, G, D), m["rot"])
    v = v.reshape(n, G, V)
    seen = window_seen(n, m["mask"]["size"])
    out = np.empty((n, H, V))
    for a in range(H):
        g = a // (H // G)
        s = m["softcap"] * np.tanh(q[:, a] @ k[:, g].T * m["scale"] / m["softcap"])
        out[:, a] = softmax_rows(s, seen) @ v[:, g]
    return (out.reshape(n, H * V) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(h, w, p, m, eps):
    return (m["left_scale"] * window_attention(h, w, p + "left.", m["left"], eps)
            + m["right_scale"] * head_delta(h, w, p + "right.", m["right"], eps))


MIXERS = {"channel_delta": channel_delta, "parallel": parallel}


# ---- feed-forward --------------------------------------------------------------------------------------------------
def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def experts(h, w, p, f):
    s = sigmoid(h @ w[p + "router"].T)
    chosen = np.argsort(-s, axis=-1, kind="stable")[:, :f["router"]["top"]]
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e in chosen[t]:
            y[t] += expert(s[t, e] * h[t], w, f"{p}e{e}.")
    return y


# ---- the model -----------------------------------------------------------------------------------------------------
def norm(x, eps, w):
    return rms(x, eps, 1.0 + w)


def forward(cfg, w, tokens, layers=None):
    """Float64 logits [n, vocab]; ``layers`` (a list) receives the residual after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        l = f"l{i}."
        x = x + MIXERS[layer["type"]](norm(x, eps, w[l + "norm1"]), w, l + "mix.", layer["mixer"], eps)
        if layer.get("mlp"):
            x = x + experts(norm(x, eps, w[l + "norm2"]), w, l + "mlp.", layer["mlp"])
        if layers is not None:
            layers.append(x)
    return norm(x, eps, w["final.norm"]) @ w["embed"].T * cfg["logit_scale"]
