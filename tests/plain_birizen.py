"""Plain, slow implementation of the Birizen decoder in float64, whole sequences, no cache.

One function per mechanism, written from the design's equations and sharing no code with the
package.  A model is (config dict, {tensor name: float64 numpy array}).

Notation: x is the residual stream [T, width]; a layer is
    x += norm1b(mixer(norm1(x)));  x += norm2b(ff(norm2(x)))
with norm(x) = x / sqrt(mean(x^2) + eps) * w.  A stretch of layers runs several times; in front of each of its passes
    x = W_in [x; x0] + step_t
with x0 the embedding output and t the number of the pass.
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


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


# ---- rotation ------------------------------------------------------------------------------------
def rot_frequencies(rot):
    """(a frequency per pair, the factor on cos and sin).  With 'scaling': pairs below lo keep their frequency, pairs
    above hi have it divided by the factor, those between go linearly from one to the other."""
    n = rot["dims"]
    base = float(rot["base"])
    f = np.array([base ** (-2.0 * i / n) for i in range(n // 2)])
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def turning(t):
        return n * math.log(sc["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo = max(math.floor(turning(sc["fast"])), 0)
    hi = min(math.ceil(turning(sc["slow"])), n - 1)
    out = f.copy()
    for i in range(n // 2):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = f[i] / sc["factor"] * r + f[i] * (1.0 - r)
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate_interleaved(x, positions, rot):
    """x [T, heads, dims], all of it turned, dimension 2i with 2i + 1."""
    f, size = rot_frequencies(rot)
    ang = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = size * np.cos(ang)[:, None, :], size * np.sin(ang)[:, None, :]
    u, v = x[..., 0::2], x[..., 1::2]
    out = np.empty_like(x)
    out[..., 0::2] = u * c - v * s
    out[..., 1::2] = v * c + u * s
    return out


# ---- mixers --------------------------------------------------------------------------------------
def fixed_decay_scan(a, k, v, q):
    """One head: S_t = a S_(t-1) + k_t v_t^T from S = 0, o_t = S_t^T q_t.  k and q [T, d], v [T, dv]."""
    S = np.zeros((k.shape[1], v.shape[1]))
    o = np.zeros((k.shape[0], v.shape[1]))
    for t in range(k.shape[0]):
        S = a * S + np.outer(k[t], v[t])
        o[t] = S.T @ q[t]
    return o


def lightning(m, W, p, h, eps):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = silu(h @ W[p + ".q"].T).reshape(T, H, d)
    k = silu(h @ W[p + ".k"].T).reshape(T, H, d)
    v = silu(h @ W[p + ".v"].T).reshape(T, H, dv)
    o = np.zeros((T, H, dv))
    for a in range(H):
        o[:, a] = fixed_decay_scan(m["decay"][a], k[:, a], v[:, a], q[:, a])
    o = rms_norm(o.reshape(T, H * dv), W[p + ".norm"], eps) * sigmoid(h @ W[p + ".g"].T)
    return o @ W[p + ".o"].T


def softmax_with_sink(s, sink):
    """Rows of scores (-inf: not seen) and one more score that only enters the sum."""
    m = np.maximum(s.max(-1, keepdims=True), sink)
    e = np.exp(s - m)
    return e / (e.sum(-1, keepdims=True) + np.exp(sink - m))


def latent_attention(m, W, p, h, eps):
    H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    pos = np.arange(T)
    q = (rms_norm(h @ W[p + ".dq"].T, W[p + ".dq.norm"], eps) @ W[p + ".uq"].T).reshape(T, H, d + r)
    down = h @ W[p + ".dkv"].T
    c = rms_norm(down[:, :R], W[p + ".dkv.norm"], eps)
    k = (c @ W[p + ".uk"].T).reshape(T, H, d)
    v = (c @ W[p + ".uv"].T).reshape(T, H, dv)
    see = pos[None, :] <= pos[:, None]
    if r:
        q_rot = rotate_interleaved(q[:, :, d:], pos, m["rot"])
        k_rot = rotate_interleaved(down[:, None, R:], pos, m["rot"])[:, 0]
    out = np.zeros((T, H, dv))
    for a in range(H):
        s = q[:, a, :d] @ k[:, a].T
        if r:
            s = s + q_rot[:, a] @ k_rot.T
        s = np.where(see, s * m["scale"], -np.inf)
        out[:, a] = softmax_with_sink(s, W[p + ".sink"][a]) @ v[:, a]
    gated = out.reshape(T, H * dv) * sigmoid(h @ W[p + ".g"].T)
    return gated @ W[p + ".o"].T


# ---- feed-forward --------------------------------------------------------------------------------
def clamped_expert(W, p, h, limit):
    g = np.minimum(h @ W[p + ".gate"].T, limit)
    u = np.clip(h @ W[p + ".up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[p + ".down"].T


def choose_experts(choice, top, groups):
    """One token's choice scores -> the chosen experts, best first (the lower index among equals).  A group counts as
    much as its two best experts together (its one expert where it has only one)."""
    n = len(choice)
    count, keep = (groups["count"], groups["keep"]) if groups else (1, 1)
    per = n // count
    value = [sum(sorted(choice[g * per:(g + 1) * per])[-2:]) for g in range(count)]
    kept = sorted(range(count), key=lambda g: (-value[g], g))[:keep]
    allowed = [e for e in range(n) if e // per in kept]
    return sorted(allowed, key=lambda e: (-choice[e], e))[:top]


def routes(router, W, p, h):
    """(chosen experts [T, top], their weights)."""
    s = sigmoid(h @ W[p + ".router"].T)
    choice = s + W[p + ".correction"]
    ids = np.array([choose_experts(c, router["top"], router.get("groups")) for c in choice])
    w = np.take_along_axis(s, ids, 1)
    return ids, w / (w.sum(-1, keepdims=True) + 1e-20)


def mixture(mlp, W, p, h):
    ids, w = routes(mlp["router"], W, p, h)
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, we in zip(ids[t], w[t]):
            y[t] += we * clamped_expert(W, f"{p}.e{e}", h[t:t + 1], mlp["expert"]["limit"])[0]
    if mlp.get("shared"):
        y = y + clamped_expert(W, p + ".shared", h, mlp["shared"]["limit"])
    return y


# ---- the model -----------------------------------------------------------------------------------
def run_order(cfg):
    """(layer, number of the pass whose first layer this is, or None)."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return ([(i, None) for i in range(a)] + [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)] +
            [(i, None) for i in range(b, n)])


def enter_pass(W, t, x, x0):
    return np.concatenate([x, x0], -1) @ W["loop.in"].T + W["loop.step"][t]


def forward(cfg, W, ids, layers_out=None):
    """Logits [T, vocab] of one whole sequence.  ``layers_out`` (a list) receives the stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x0 = W["embed"][np.asarray(ids)]
    x = x0
    for i, t in run_order(cfg):
        if t is not None:
            x = enter_pass(W, t, x, x0)
        L, p = cfg["layers"][i], f"l{i}"
        mixer = {"lightning": lightning, "latent_attention": latent_attention}[L["type"]]
        y = mixer(L["mixer"], W, p + ".mix", rms_norm(x, W[p + ".norm1"], eps), eps)
        x = x + rms_norm(y, W[p + ".norm1b"], eps)
        if L.get("mlp") is not None:
            y = mixture(L["mlp"], W, p + ".mlp", rms_norm(x, W[p + ".norm2"], eps))
            x = x + rms_norm(y, W[p + ".norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, W["final.norm"], eps) @ W["embed"].T


def greedy(cfg, W, ids, n):
    """n tokens by arg-max, each from a whole forward pass."""
    ids, out = list(ids), []
    for _ in range(n):
        out.append(int(np.argmax(forward(cfg, W, ids)[-1])))
        ids.append(out[-1])
    return out
