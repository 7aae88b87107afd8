"""Small Tupalorn configurations, model folders with random weights, and the plain implementation's logits."""
import torch

import plain_tupalorn as plain


def m2(heads, vdim, state, groups, conv, norm_groups):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}}


def ret(dim, vdim, decay, rot_dims, base):
    return {"type": "retention", "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay),
                                           "rot": {"dims": rot_dims, "base": base}}}


def att(heads, kv_heads, dim, vdim, scale, window, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def layer(mixer, ff, limit=1.0):
    return dict(mixer, mlp={"kind": "dense", "ff": ff, "limit": limit} if ff else None)


def model(vocab, width, eps, softcap, layers):
    return {"architecture": "Tupalorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": softcap, "layers": layers}


# Odd sizes throughout: heads that fill no multiple of 16, an odd value head, more groups than one, norm parts that are
# neither heads nor groups, a short convolution, a window of one position, one layer's keys and values read by a layer that
# sees further back than it does and by one that sees less far, layers without a feed-forward.
ODD = model(211, 72, 1e-5, 20.0, [
    layer(m2(6, 20, 24, 3, 4, 2), 100, 1.5),
    layer(att(6, 3, 24, 40, 0.5, 12), 64, 0.8),
    layer(ret(24, 15, (0.9, 0.97, 0.995, 0.5, 0.999), 8, 500.0), None),
    layer(att(6, 3, 24, 40, 0.4, 29, kv_from=1), 48, 3.0),
    layer(att(4, 4, 16, 16, 0.6, 1), 56, 1.0),
    layer(m2(3, 17, 5, 1, 2, 3), 40, 0.5),
    layer(att(6, 3, 24, 40, 0.5, 5, kv_from=1), None),
])
# Sizes the tensor-core kernels take, value heads of several tiles, states and key heads of more than one tile, a
# convolution of three taps, a window longer than a portion.
WIDE = model(1032, 256, 1e-6, 50.0, [
    layer(ret(64, 128, (0.93, 0.99, 0.998, 0.9995), 32, 25000.0), 512, 2.5),
    layer(att(8, 2, 64, 64, 0.25, 48), 256, 1.5),
    layer(m2(8, 64, 128, 2, 4, 1), 512, 1.0),
    layer(att(4, 1, 128, 128, 0.2, 208), 256, 4.0),
    layer(att(8, 2, 64, 64, 0.25, 80, kv_from=1), 264, 1.0),
    layer(m2(2, 96, 144, 1, 3, 4), None),
    layer(ret(256, 48, (0.96, 0.9999), 256, 10000.0), 128, 1.0),
])
# A width that is no multiple of 8 (no tensor-core product takes it), one head, a convolution of one tap (no carried
# inputs), many taps, a window longer than any request, no rotation at all, a decay of one.
THIN = model(97, 44, 1e-4, 8.0, [
    layer(ret(6, 10, (1.0,), 2, 77.0), 24, 1.0),
    layer(m2(2, 11, 7, 2, 1, 1), 20, 2.0),
    layer(att(2, 1, 20, 12, 0.7, 500), None),
    layer(m2(4, 6, 9, 2, 7, 4), 20, 0.7),
    layer(ret(9, 3, (0.8, 0.99), 0, 50.0), None),
])
CONFIGS = {"odd": ODD, "wide": WIDE, "thin": THIN}
BLOCKS = {"odd": 8, "wide": 16, "thin": 4}


def make_folder(cfg_dict, folder, seed, dtype=torch.float32, edit=None):
    """A model folder with random weights: norm weights, biases and the state-space parameters well away from their neutral
    values, decays of the recurrences spread from those that forget in a token to those that hold hundreds."""
    from hfcpu_b200.config import config_from_dict
    from hfcpu_b200.models import build_model_specs
    from hfcpu_b200.weights import random_tensors, write_safetensors, weights_path
    cfg = config_from_dict(cfg_dict)
    cfg.save(folder)
    soft = dtype == torch.bfloat16
    tensors = random_tensors(build_model_specs(cfg), seed, torch.float32, std=0.06 if soft else 0.1)
    g = torch.Generator().manual_seed(seed)
    uni = lambda t, lo, hi: torch.empty(t.shape).uniform_(lo, hi, generator=g)
    for name in tensors:
        t = tensors[name]
        if name == "embed":
            tensors[name] = t * (6 if soft else 8)
        elif name.endswith((".q.norm", ".k.norm")):
            tensors[name] = uni(t, 0.6, 1.8)
        elif name.endswith(("norm1", "final.norm", ".norm")):
            tensors[name] = uni(t, 0.5, 1.6)
        elif name.endswith(".conv"):
            tensors[name] = uni(t, -1.0, 1.0)
        elif name.endswith("A_log"):
            tensors[name] = uni(t, -4.0, 1.0)
        elif name.endswith("dt_bias"):
            tensors[name] = uni(t, -4.0, 0.5)
        elif name.endswith(".D"):
            tensors[name] = uni(t, -1.5, 1.5)
        elif name.endswith(".b"):
            tensors[name] = uni(t, -0.7, 0.7)
        elif name.endswith((".gate", ".up", ".mix.in", ".mix.g", ".mix.o", ".down")):
            tensors[name] = t * 1.5
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
