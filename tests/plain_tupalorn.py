"""Plain, slow implementation of the Tupalorn decoder in float64, whole sequences, no cache.

One function per mechanism, written from the design's equations and sharing no code with the
package.  A model is (config dict, {tensor name: float64 numpy array}).

Notation: x is the residual stream [T, width]; a layer is
    h = layernorm(x);  x += mixer(h) + ff(h)
with layernorm(x) = (x - mean) / sqrt(var + eps) * w (no bias): both sublayers read the same h.
"""
import json
import math
import os
import struct

import numpy as np


# ---- files ---------------------------------------------------------------------------------------
def read_safetensors(path):
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        head = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, m in head.items():
        if name == "__metadata__":
            continue
        a, b = m["data_offsets"]
        raw = data[a:b]
        if m["dtype"] == "BF16":
            v = (np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16).view(np.float32)
        elif m["dtype"] == "F32":
            v = np.frombuffer(raw, dtype="<f4")
        elif m["dtype"] == "I32":
            v = np.frombuffer(raw, dtype="<i4")
        else:
            raise ValueError(m["dtype"])
        out[name] = v.astype(np.float64).reshape(m["shape"])
    return out


def read_folder(folder):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(folder, "model.safetensors"))


# ---- element-wise --------------------------------------------------------------------------------
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def softmax_rows(s):
    """Softmax over the last axis; entries of -inf get weight zero."""
    m = s.max(-1, keepdims=True)
    e = np.exp(s - m)
    return e / e.sum(-1, keepdims=True)


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


# ---- norms ---------------------------------------------------------------------------------------
def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * w


def unit_rms(x, eps):
    """Last axis divided by its root mean square."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def rms_norm_parts(x, w, parts, eps):
    """The last axis in equal parts, each divided by its own root mean square; one weight over all of it."""
    T, n = x.shape
    return unit_rms(x.reshape(T, parts, n // parts), eps).reshape(T, n) * w


# ---- rotation ------------------------------------------------------------------------------------
def rotate_half_layout(x, positions, rot):
    """x [T, heads, D]: the first rot.dims dimensions of each head turn, dimension i with i + dims/2."""
    n = rot["dims"]
    half = n // 2
    f = np.array([float(rot["base"]) ** (-2.0 * i / n) for i in range(half)])
    ang = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    u, v = x[..., :half], x[..., half:n]
    out = x.copy()
    out[..., :half] = u * c - v * s
    out[..., half:n] = v * c + u * s
    return out


# ---- convolution over time -----------------------------------------------------------------------
def causal_conv(x, w, b):
    """Per channel: y_t = b + sum_j w[:, j] x_(t - taps + 1 + j), zeros before the start."""
    T, C = x.shape
    taps = w.shape[1]
    pad = np.concatenate([np.zeros((taps - 1, C)), x], 0)
    y = np.tile(b, (T, 1))
    for j in range(taps):
        y = y + w[:, j] * pad[j:j + T]
    return y


# ---- the recurrence ------------------------------------------------------------------------------
def scalar_decay_scan(a, k, u, q):
    """One head: S_t = a_t S_(t-1) + k_t u_t^T from S = 0, o_t = S_t^T q_t.  a [T], k and q [T, d], u [T, dv]."""
    T = k.shape[0]
    S = np.zeros((k.shape[1], u.shape[1]))
    o = np.zeros((T, u.shape[1]))
    for t in range(T):
        S = a[t] * S + np.outer(k[t], u[t])
        o[t] = S.T @ q[t]
    return o


# ---- mixers --------------------------------------------------------------------------------------
def mamba2(m, W, p, h, eps):
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    T = h.shape[0]
    row = h @ W[p + ".in"].T
    z, xbc, dt = row[:, :inner], row[:, inner:inner + inner + 2 * G * N], row[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, W[p + ".conv"], W[p + ".conv.b"]))
    x = xbc[:, :inner].reshape(T, H, dv)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + W[p + ".dt_bias"])
    y = np.zeros((T, H, dv))
    for a in range(H):
        g = a // (H // G)
        decay = np.exp(-np.exp(W[p + ".A_log"][a]) * dt[:, a])
        y[:, a] = scalar_decay_scan(decay, B[:, g], dt[:, a:a + 1] * x[:, a], C[:, g]) + W[p + ".D"][a] * x[:, a]
    y = rms_norm_parts(y.reshape(T, inner) * silu(z), W[p + ".norm"], m["norm_groups"], eps)
    return y @ W[p + ".o"].T


def retention(m, W, p, h, eps):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    pos = np.arange(T)
    q = rotate_half_layout((h @ W[p + ".q"].T).reshape(T, H, d), pos, m["rot"])
    k = rotate_half_layout((h @ W[p + ".k"].T).reshape(T, H, d), pos, m["rot"]) * d ** -0.5
    v = (h @ W[p + ".v"].T).reshape(T, H, dv)
    o = np.zeros((T, H, dv))
    for a in range(H):
        o[:, a] = scalar_decay_scan(np.full(T, m["decay"][a]), k[:, a], v[:, a], q[:, a])
    o = unit_rms(o, eps).reshape(T, H * dv) * silu(h @ W[p + ".g"].T)
    return o @ W[p + ".o"].T


def window_mask(T, size):
    """[T, T] True where query i sees key j: itself and the size - 1 keys before it."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (i - j < size)


def attention_keys_values(m, W, p, h, eps):
    T = h.shape[0]
    G, d, dv = m["kv_heads"], m["dim"], m["vdim"]
    k = rms_norm(h @ W[p + ".k"].T, W[p + ".k.norm"], eps).reshape(T, G, d)
    v = (h @ W[p + ".v"].T).reshape(T, G, dv)
    return k, v


def attention(m, W, p, h, eps, kv):
    """Grouped heads, query norm over the whole projection, no rotation, a window, one sigmoid gate per head.  ``kv``: the
    keys and values attended over (this layer's own or an earlier layer's)."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(h @ W[p + ".q"].T, W[p + ".q.norm"], eps).reshape(T, H, d)
    k, v = kv
    see = window_mask(T, m["mask"]["size"])
    gate = sigmoid(h @ W[p + ".g"].T)
    out = np.zeros((T, H, dv))
    for a in range(H):
        g = a // (H // G)
        s = np.where(see, (q[:, a] @ k[:, g].T) * m["scale"], -np.inf)
        out[:, a] = softmax_rows(s) @ v[:, g] * gate[:, a:a + 1]
    return out.reshape(T, H * dv) @ W[p + ".o"].T


# ---- feed-forward --------------------------------------------------------------------------------
def clamped_ff(mlp, W, p, h):
    """g = min(Wg h + bg, limit), u = clamp(Wu h + bu, -limit, limit); down(g sigmoid(1.702 g) (u + 1)) + b."""
    lim = mlp["limit"]
    g = np.minimum(h @ W[p + ".gate"].T + W[p + ".gate.b"], lim)
    u = np.clip(h @ W[p + ".up"].T + W[p + ".up.b"], -lim, lim)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[p + ".down"].T + W[p + ".down.b"]


# ---- the model -----------------------------------------------------------------------------------
def forward(cfg, W, ids, layers_out=None):
    """Logits [T, vocab] of one whole sequence.  ``layers_out`` (a list) receives the stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(ids)]
    kvs = {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}", L["mixer"]
        h = layer_norm(x, W[p + ".norm1"], eps)
        if L["type"] == "mamba2":
            y = mamba2(m, W, p + ".mix", h, eps)
        elif L["type"] == "retention":
            y = retention(m, W, p + ".mix", h, eps)
        elif L["type"] == "attention":
            j = m.get("kv_from")
            if j is None:
                kvs[i] = attention_keys_values(m, W, p + ".mix", h, eps)
            y = attention(m, W, p + ".mix", h, eps, kvs[i if j is None else j])
        else:
            raise ValueError(L["type"])
        if L.get("mlp") is not None:
            y = y + clamped_ff(L["mlp"], W, p + ".mlp", h)
        x = x + y
        if layers_out is not None:
            layers_out.append(x.copy())
    logits = layer_norm(x, W["final.norm"], eps) @ W["embed"].T
    return soft_cap(logits, cfg["logit_softcap"])


def greedy(cfg, W, ids, n):
    """n tokens by arg-max, each from a whole forward pass."""
    ids, out = list(ids), []
    for _ in range(n):
        out.append(int(np.argmax(forward(cfg, W, ids)[-1])))
        ids.append(out[-1])
    return out
