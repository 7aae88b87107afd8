"""Small Birizen configurations, model folders with random weights, and the plain implementation's logits."""
import torch

import plain_birizen as plain


def lightning(dim, vdim, decay):
    return {"type": "lightning", "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base=100.0, scaling=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if rot_dim:
        m["rot"] = {"dims": rot_dim, "base": base}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": m}


def moe(experts, top, ff, limit, groups=None, shared=None):
    """``shared`` = (ff, limit)."""
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": r}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def layer(mixer, mlp):
    return dict(mixer, mlp=mlp)


def model(vocab, width, eps, layers, loop=None):
    d = {"architecture": "Birizen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# Odd sizes throughout: heads that fill no multiple of 16, odd value heads, a loop in the middle of the layers, layers with
# no feed-forward at the end of a pass and at the end of the model, limits of every size, groups of three, rows of latents
# that are no multiple of 8.
ODD = model(211, 72, 1e-5, [
    layer(lightning(20, 15, (0.9, 0.98, 0.999, 0.4, 1.0)), moe(9, 3, 40, 0.6, (3, 2), (56, 1.1))),
    layer(latent(6, 24, 10, 20, 28, 30, 0.4, 100.0, (3.0, 64, 8.0, 1.0)), moe(6, 2, 24, 1.4, None, (24, 0.5))),
    layer(lightning(24, 40, (0.97, 0.7)), None),
    layer(latent(3, 12, 6, 33, 40, 18, 0.6, 2000.0), moe(8, 4, 36, 0.9, (4, 2))),
    layer(lightning(9, 12, (0.995, 0.6, 0.85)), None),
], (1, 3, 2))
# Sizes the tensor-core kernels take: latent rows of 128 and 64 (the tiled attention kernels), value heads of several tiles, a
# loop at the start that runs three times, a loop's layer after which nothing but one layer follows.
WIDE = model(1032, 256, 1e-6, [
    layer(latent(8, 64, 32, 64, 96, 96, 0.15, 10000.0, (8.0, 128, 16.0, 1.0)), moe(8, 2, 64, 1.0, (4, 2), (128, 2.0))),
    layer(lightning(64, 128, (0.93, 0.99, 0.998, 0.9995)), moe(16, 4, 48, 2.5, (4, 3), (96, 0.7))),
    layer(latent(4, 32, 16, 96, 64, 48, 0.2, 500.0), moe(4, 1, 128, 1.5, (2, 1))),
], (0, 2, 3))
# A width that is no multiple of 8 (no tensor-core product takes it), one head, no rotated part, ranks of a few values, a
# loop that runs once and ends the model, groups of one expert, every group kept, every expert chosen.
THIN = model(97, 44, 1e-4, [
    layer(lightning(6, 10, (0.8,)), moe(4, 2, 12, 0.8, (4, 3), (20, 0.8))),
    layer(latent(1, 7, 0, 5, 3, 9, 0.9), moe(3, 3, 20, 2.0)),
    layer(lightning(5, 3, (0.99, 0.5)), moe(6, 2, 16, 0.7, (2, 2), (8, 3.0))),
], (1, 3, 1))
# No loop at all.
FLAT = model(64, 48, 1e-5, [
    layer(latent(2, 16, 8, 16, 24, 24, 0.5, 50.0, (2.0, 32, 4.0, 1.0)), None),
    layer(lightning(16, 16, (0.95, 0.999)), moe(4, 2, 32, 1.0, (2, 1), (32, 1.0))),
])
# Latent attention only (no state at all; launches may overlap), with a loop around the last of two layers.
LATENT = model(130, 128, 1e-6, [
    layer(latent(4, 32, 16, 32, 48, 48, 0.3, 1000.0, (4.0, 64, 8.0, 2.0)), moe(8, 3, 32, 1.0, (4, 2), (64, 1.5))),
    layer(latent(2, 24, 8, 40, 32, 32, 0.4, 200.0), moe(4, 2, 40, 0.8, None, (48, 0.8))),
], (1, 2, 2))
CONFIGS = {"odd": ODD, "wide": WIDE, "thin": THIN, "flat": FLAT, "latent": LATENT}
BLOCKS = {"odd": 8, "wide": 16, "thin": 4, "flat": 8, "latent": 8}


def make_folder(cfg_dict, folder, seed, dtype=torch.float32, edit=None, sharp=2.5):
    """A model folder with random weights in which every mechanism matters: attention far from uniform, sinks of both signs,
    routers that decide clearly with corrections that change choices, clamps at work, norm weights away from one, passes
    that differ.  Stored in bfloat16 the scores are milder, so that their rounding does not swamp the comparison."""
    from hfcpu_b200.config import config_from_dict
    from hfcpu_b200.models import build_model_specs
    from hfcpu_b200.weights import random_tensors, write_safetensors, weights_path
    cfg = config_from_dict(cfg_dict)
    cfg.save(folder)
    soft = dtype == torch.bfloat16
    tensors = random_tensors(build_model_specs(cfg), seed, torch.float32, std=1.0)
    g = torch.Generator().manual_seed(seed)
    uni = lambda t, lo, hi: torch.empty(t.shape).uniform_(lo, hi, generator=g)
    for name in tensors:
        t = tensors[name]
        if name.endswith(("norm", "norm1", "norm2", "norm1b", "norm2b")):
            tensors[name] = uni(t, 0.5, 1.5)
        elif name.endswith(".sink"):
            tensors[name] = uni(t, -2.0, 2.0)
        elif name.endswith(".correction"):
            # most choice scores near or below zero; stored in bfloat16 they lie so far apart that close calls are rare (a choice
            # that flips with rounding changes a row, and all later rows through the states, by more than rounding does)
            tensors[name] = -0.25 * torch.randperm(t.shape[0], generator=g).float() + uni(t, 0.0, 0.02) if soft else uni(t, -0.7, 0.1)
        elif name.endswith("loop.step"):
            tensors[name] = t * 0.7
        elif name == "embed":
            tensors[name] = t * 1.2
        else:
            gain = 1.0
            if name.endswith(".router"):
                gain = 0.35 if soft else 1.5
            elif name.endswith(".uq"):
                gain = 1.0 if soft else sharp
            tensors[name] = t * gain / t.shape[1] ** 0.5
    if edit:
        edit(tensors)
    # what is stored is what both sides read: round once to the storage type
    write_safetensors(weights_path(folder), {k: v.to(dtype) for k, v in tensors.items()})
    return folder


_PLAIN = {}


def plain_logits(folder, ids):
    key = (folder, tuple(ids))
    if key not in _PLAIN:
        cfg, W = plain.read_folder(folder)
        _PLAIN[key] = torch.from_numpy(plain.forward(cfg, W, list(ids)))
    return _PLAIN[key]


def requests(vocab, lengths, seed=0):
    g = torch.Generator().manual_seed(seed)
    return {f"r{i}": torch.randint(0, vocab, (n,), generator=g).tolist() for i, n in enumerate(lengths)}


def far_folder(spec, folder, dtype, n, place, far, last, vocab=150, width=96):
    """A one-layer model in which what token ``far`` at position ``place`` leaves behind decides what the query of token
    ``last`` at position n - 1 gets, whatever lies between.  Lightning: the keys of all other tokens are zero (their embeddings
    have no part along the key projection).  Latent attention: the far token's rotated key part is the sum of the last
    query's rotated parts turned by the distance between the two, and that score stands out."""
    cfg = model(vocab, width, 1e-5, [layer(spec, None)])
    m = spec["mixer"]

    def edit(t):
        W = {k: v.double().numpy() for k, v in t.items()}
        import numpy as np
        if spec["type"] == "lightning":
            rows = W["l0.mix.k"] * W["l0.norm1"]
            basis = np.linalg.qr(rows.T)[0]
            e = W["embed"] - (W["embed"] @ basis) @ basis.T
            e[far] = W["embed"][far]
        else:
            t["l0.mix.sink"].fill_(-1.0)
            h = plain.rms_norm(W["embed"][last][None], W["l0.norm1"], 1e-5)
            cq = plain.rms_norm(h @ W["l0.mix.dq"].T, W["l0.mix.dq.norm"], 1e-5)
            q = (cq @ W["l0.mix.uq"].T).reshape(1, m["heads"], m["dim"] + m["rot_dim"])[..., m["dim"]:]
            u = plain.rotate_interleaved(q, [n - 1 - place], m["rot"]).sum(1)[0]
            e = W["embed"].copy()
            d = (W["l0.mix.dkv"][m["kv_rank"]:].T @ u) * W["l0.norm1"]
            e[far] = d / np.linalg.norm(d) * np.linalg.norm(e[last])
            t["l0.mix.dkv"][m["kv_rank"]:] *= 2.0
        t["embed"].copy_(torch.from_numpy(e))
    return make_folder(cfg, folder, 23, dtype, edit=edit, sharp=3.0)
