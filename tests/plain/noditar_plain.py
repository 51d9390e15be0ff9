"""A plain, slow Noditar forward pass: one whole sequence from position 0, no cache, one function per mechanism.

It shares no code with ``purhie_b200``: it reads ``config.json`` with ``json`` and the weight file by its byte
layout, and states every equation directly.  Everything runs in float64.

The design in short (names of config.json in quotes):

* The residual is "streams" rows per token, X[0 .. s-1], each the token's embedding at first.  A part f (a mixer or a
  feed-forward) with the vectors a, b and the matrix M of its own reads u = sum_s a[s] X[s], gives y = f(rms(u; norm)),
  and every stream becomes X'[t] = sum_s M[s, t] X[s] + b[t] y.  Behind the last layer the streams are added up.
* Mixer "latent_attention": c = rms(W_dkv h; dkv.norm) is all a token leaves behind; per head k = W_uk c, v = W_uv c,
  score (q . k) * "scale", softmax over every earlier position, the heads side by side times sigmoid(W_g h), W_o.
* Mixer "attention": grouped heads, q and k over their root mean square per head, score (q . k) * "scale" minus
  2^(-8 (h + 1) / H) times the distance, weights exp(s_j) / (1 + sum exp(s)), the same gate, W_o.
* Mixer "mamba2": [z | x | B | C | dt] = W_in h; x, B and C through a causal convolution per channel and silu;
  dt = softplus(dt + dt_bias); per head S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x; y * silu(z) RMS-normed in
  "norm_groups" parts; W_o.
* Feed-forward "dense": g = min(W_gate h, limit), u = clamp(W_up h, +-limit), W_down (g sigmoid(1.702 g) (u + 1)).
* logits = head rms(x; final.norm).
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


def causal(n):
    """[n, n] True where query i sees key j."""
    return np.arange(n)[:, None] >= np.arange(n)[None, :]


# ---- the streams ---------------------------------------------------------------------------------------------------
def streams_read(X, a):
    """X [streams, n, width] -> u [n, width] = sum_s a[s] X[s]."""
    return np.tensordot(a, X, axes=(0, 0))


def streams_update(X, M, b, y):
    """X'[t] = sum_s M[s, t] X[s] + b[t] y."""
    return np.stack([sum(M[s, t] * X[s] for s in range(X.shape[0])) + b[t] * y for t in range(X.shape[0])])


# ---- mixers --------------------------------------------------------------------------------------------------------
def softmax_rows(s, seen, sink=False):
    """Softmax over the keys a row sees; with a sink, one is added to the denominator."""
    s = np.where(seen, s, -np.inf)
    top = s.max(axis=-1, keepdims=True)
    if sink:
        top = np.maximum(top, 0.0)
    e = np.exp(s - top)
    return e / (e.sum(axis=-1, keepdims=True) + (np.exp(-top) if sink else 0.0))


def latent_attention(h, w, p, m, eps):
    n = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(n, H, D)
    c = rms(h @ w[p + "dkv"].T, eps, w[p + "dkv.norm"])
    k = (c @ w[p + "uk"].T).reshape(n, H, D)
    v = (c @ w[p + "uv"].T).reshape(n, H, V)
    out = np.empty((n, H, V))
    for a in range(H):
        out[:, a] = softmax_rows(q[:, a] @ k[:, a].T * m["scale"], causal(n)) @ v[:, a]
    return (out.reshape(n, H * V) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def head_slopes(H):
    return 2.0 ** (-8.0 * (np.arange(H) + 1) / H)


def biased_attention(h, w, p, m, eps, sink=True, slopes=None):
    n = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ w[p + "q"].T).reshape(n, H, D), eps)
    k = rms((h @ w[p + "k"].T).reshape(n, G, D), eps)
    v = (h @ w[p + "v"].T).reshape(n, G, V)
    distance = np.arange(n)[:, None] - np.arange(n)[None, :]
    slopes = head_slopes(H) if slopes is None else slopes
    out = np.empty((n, H, V))
    for a in range(H):
        g = a // (H // G)
        s = q[:, a] @ k[:, g].T * m["scale"] - slopes[a] * distance
        out[:, a] = softmax_rows(s, causal(n), sink) @ v[:, g]
    return (out.reshape(n, H * V) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def causal_conv(x, taps, bias):
    """x [n, channels]: y_i = bias + sum_j taps[:, j] x_(i - K + 1 + j), zeros before the start."""
    K = taps.shape[1]
    pad = np.concatenate([np.zeros((K - 1, x.shape[1])), x])
    return bias + sum(taps[:, j] * pad[j:j + x.shape[0]] for j in range(K))


def state_space_scan(x, B, C, dt, decay, D, heads_per_group):
    """x [n, H, P], B and C [n, G, N], dt and decay [n, H] -> y [n, H, P], token by token from S = 0 ([H, N, P])."""
    n, H, P = x.shape
    S = np.zeros((H, B.shape[2], P))
    group = np.arange(H) // heads_per_group
    y = np.empty_like(x)
    for t in range(n):
        S = decay[t][:, None, None] * S + dt[t][:, None, None] * B[t][group][:, :, None] * x[t][:, None, :]
        y[t] = np.einsum("hnp,hn->hp", S, C[t][group]) + D[:, None] * x[t]
    return y


def mamba2(h, w, p, m, eps):
    n = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    u = h @ w[p + "in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:inner + inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x = xbc[:, :inner].reshape(n, H, P)
    B = xbc[:, inner:inner + G * N].reshape(n, G, N)
    C = xbc[:, inner + G * N:].reshape(n, G, N)
    dt = softplus(dt + w[p + "dt_bias"])
    y = state_space_scan(x, B, C, dt, np.exp(-np.exp(w[p + "A_log"]) * dt), w[p + "D"], H // G)
    y = (y.reshape(n, inner) * silu(z)).reshape(n, m["norm_groups"], -1)
    return (rms(y, eps).reshape(n, inner) * w[p + "norm"]) @ w[p + "o"].T


MIXERS = {"latent_attention": latent_attention, "attention": biased_attention, "mamba2": mamba2}


# ---- feed-forward --------------------------------------------------------------------------------------------------
def clamped_unit(h, w, p, limit):
    g = np.minimum(h @ w[p + "gate"].T, limit)
    u = np.clip(h @ w[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


# ---- the model -----------------------------------------------------------------------------------------------------
def forward(cfg, w, tokens, layers=None):
    """Float64 logits [n, vocab]; ``layers`` (a list) receives the sum of the streams after every layer."""
    eps = cfg["norm"]["eps"]
    X = np.stack([w["embed"][np.asarray(tokens)]] * cfg["streams"])

    def part(X, l, q, f):
        u = streams_read(X, w[f"{l}hc{q}.in"])
        return streams_update(X, w[f"{l}hc{q}.mix"], w[f"{l}hc{q}.out"], f(rms(u, eps, w[f"{l}norm{q}"])))

    for i, layer in enumerate(cfg["layers"]):
        l = f"l{i}."
        X = part(X, l, 1, lambda h: MIXERS[layer["type"]](h, w, l + "mix.", layer["mixer"], eps))
        if layer.get("mlp"):
            X = part(X, l, 2, lambda h: clamped_unit(h, w, l + "mlp.", layer["mlp"]["limit"]))
        if layers is not None:
            layers.append(X.sum(axis=0))
    return rms(X.sum(axis=0), eps, w["final.norm"]) @ w["head"].T
