"""Tupalorn on the GPU: each mechanism's kernels alone against the plain implementation's functions, then the engine under
every way of cutting the work, pages and slots used again, keys just inside and just outside every window in prompts and in
decoding, far keys through the recurrences' states, long decoding, and greedy generation through the entry point and the
trace program."""
import os
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_tupalorn as plain
import traces
from tupalorn_util import BLOCKS, CONFIGS, att, layer, m2, make_folder, model, plain_logits, requests, ret

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL = {"float32": 2e-4, "bfloat16": 3e-2}
# two runs of the engine against each other; in bfloat16 they take different kernels (tiles, chunks of the recurrence,
# single tokens), each of which is within TOL of the exact result
SELF_TOL = {"float32": 4e-5, "bfloat16": 3e-2}
KTOL = {"float32": 3e-6, "bfloat16": 8e-3}          # one kernel's output against float64


def K():
    from hfcpu_b200 import kernels
    return kernels


def dev(a, dtype=torch.float32):
    return torch.as_tensor(np.asarray(a), dtype=torch.float64).to(dtype).to(DEV).contiguous()


def f64(t):
    return t.double().cpu().numpy()


def rel(a, b):
    b = torch.as_tensor(np.asarray(b), dtype=torch.float64)
    return float((a.double().cpu() - b).abs().max() / b.abs().max().clamp_min(1e-30))


def rng(seed):
    return np.random.default_rng(seed)


def step_ctx(parts, dtype=torch.float32, positions=None):
    """The step's index arrays for [(slot, number of tokens)]."""
    from hfcpu_b200.engine.step import Workspace
    lens = [n for _, n in parts]
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    arrays = {k: i32(v) for k, v in K().decay_chunk_arrays(lens).items()}
    return SimpleNamespace(token_seq=i32(np.repeat(np.arange(len(parts)), lens)), cu_tokens=i32(np.cumsum([0] + lens)),
                           seq_slots=i32([s for s, _ in parts]), num_seqs=len(parts), max_q_len=max(lens), run_dtype=dtype,
                           positions=None if positions is None else i32(positions), arrays=lambda key: arrays,
                           buf=Workspace(torch.device(DEV)).get)


def padded(x, heads, dtype):
    """x [T, heads, n] as the recurrence takes it: zeros behind every head up to a multiple of 16."""
    T, _, n = x.shape
    out = np.zeros((T, heads, K().padded_head(n)))
    out[..., :n] = x
    return dev(out.reshape(T, -1), dtype)


# ---- each mechanism alone ---------------------------------------------------------------------------
# (heads, query/key heads, d, dv): one tile and several, odd value heads, one head for all queries and one each
SCAN_GEOMS = [(4, 4, 64, 128), (6, 2, 24, 15), (3, 1, 5, 17), (8, 1, 128, 64), (2, 2, 256, 48), (2, 1, 144, 96), (1, 1, 300, 20), (5, 5, 16, 16)]


@pytest.mark.parametrize("form", ["walk float32", "walk bfloat16", "chunks"])
@pytest.mark.parametrize("geom", SCAN_GEOMS)
def test_recurrence_across_steps(geom, form):
    """Three requests over slots in scrambled order, cut so that portions end just before, at and just behind a chunk's edge,
    beside single tokens and short portions: outputs and the state that is left.  Decays from one that forgets at once to
    one that forgets nothing; step sizes and the skip term present or not."""
    H, Hq, d, dv = geom
    r = rng(sum(geom))
    dt = torch.float32 if form == "walk float32" else torch.bfloat16
    per_token = Hq != H
    cuts = [[(0, 64), (2, 1)], [(0, 63), (1, 130), (2, 2)], [(0, 65)], [(1, 1), (0, 1)], [(1, 17), (2, 15), (0, 16)]]
    total = {s: sum(n for c in cuts for q, n in c if q == s) for s in range(3)}
    slot = {0: 2, 1: 0, 2: 3}
    data = {}
    for s, n in total.items():
        rnd = lambda *sh: f64(dev(r.standard_normal(sh), dt))
        la = -np.exp(r.uniform(-6, 2, (n, H)) if per_token else r.uniform(-7, 0, H)[None].repeat(n, 0))
        data[s] = {"q": rnd(n, Hq, d), "k": rnd(n, Hq, d) * d ** -0.5, "u": rnd(n, H, dv), "la": la, "c": r.uniform(0.01, 1.5, (n, H))}
        data[s]["k"] = f64(dev(data[s]["k"], dt))
    if not per_token:
        for s in data:
            data[s]["la"] = data[0]["la"][:1].repeat(total[s], 0)
            data[s]["la"][:, 0] = 0.0                       # a head that forgets nothing
    skip = r.uniform(-1, 1, H) if per_token else None
    want = {}
    for s, n in total.items():
        e = data[s]
        want[s] = np.stack([plain.scalar_decay_scan(np.exp(e["la"][:, a]), e["k"][:, a // (H // Hq)],
                                                    e["u"][:, a] * (e["c"][:, a:a + 1] if per_token else 1.0), e["q"][:, a // (H // Hq)])
                            + (skip[a] * e["u"][:, a] if per_token else 0.0) for a in range(H)], 1)
    dp, dvp = K().padded_head(d), K().padded_head(dv)
    state = torch.zeros(4, H, dvp, dp, dtype=torch.float32, device=DEV)
    state[1] = 7.0                                           # somebody else's
    got, at = {s: [] for s in total}, {s: 0 for s in total}
    for cut in cuts:
        ctx = step_ctx([(slot[s], n) for s, n in cut], dt)
        take = lambda name: np.concatenate([data[s][name][at[s]:at[s] + n] for s, n in cut])
        q, k, u = padded(take("q"), Hq, dt), padded(take("k"), Hq, dt), padded(take("u"), H, dt)
        T = q.shape[0]
        la = dev(take("la")) if per_token else dev(data[0]["la"][0])
        o = torch.full((T, H * dv), float("nan"), dtype=torch.float32, device=DEV)
        K().decay_scan(q, k, u, la, dev(take("c")) if per_token else None, None if skip is None else dev(skip), state, ctx, o, H, Hq, d, dv,
                       chunks=ctx.arrays(None) if form == "chunks" else None)
        b = 0
        for s, n in cut:
            got[s].append(o[b:b + n].view(n, H, dv))
            b += n
            at[s] += n
    tol = 2e-5 if form != "chunks" else 1e-4                 # chunks: operands as two bfloat16 pieces
    for s in total:
        assert rel(torch.cat(got[s]), want[s]) < tol, s
    assert bool((state[1] == 7.0).all()) and bool((state[0, :, dv:] == 0).all()) and bool((state[0, :, :, d:] == 0).all())
    K().check_device_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("geom", [(6, 3, 24, 20, 4), (3, 1, 5, 17, 2), (2, 2, 7, 11, 1), (4, 2, 9, 6, 7), (8, 1, 128, 64, 4), (2, 1, 16, 8, 16)])
def test_state_space_operands_across_steps(dtype, geom):
    """The convolution with its carried inputs over several steps (portions shorter than the taps among them), silu, the step
    sizes and the logarithms of the decays; a slot that is used again starts from zeros."""
    H, G, d, dv, taps = geom
    dt, r = DT[dtype], rng(sum(geom))
    inner, C = H * dv, H * dv + 2 * G * d
    row = (inner + C + H + 7) // 8 * 8
    w, b = dev(r.uniform(-1, 1, (C, taps)), dt), dev(r.uniform(-1, 1, C), dt)
    dtb, rate = dev(r.uniform(-3, 1, H), dt), dev(np.exp(r.uniform(-3, 1, H)))
    carried = torch.zeros(3, max(taps - 1, 1), C, dtype=torch.float32, device=DEV)
    x = {s: r.standard_normal((n, row)) for s, n in ((0, 61), (1, 12), (2, 40))}
    got, at = {s: [] for s in x}, {s: 0 for s in x}
    for cut in [[(0, 1), (2, 1)], [(0, 2), (1, 3)], [(0, 1), (1, 1), (2, 1)], [(2, 38), (0, 40), (1, 1)], [(0, 17), (1, 7)]]:
        ctx = step_ctx([(s, n) for s, n in cut], dt)
        src = dev(np.concatenate([x[s][at[s]:at[s] + n] for s, n in cut]))
        T = src.shape[0]
        q, k = (torch.full((T, G * K().padded_head(d)), 3.0, dtype=dt, device=DEV) for _ in range(2))
        u = torch.full((T, H * K().padded_head(dv)), 3.0, dtype=dt, device=DEV)
        step, la = torch.empty(T, H, device=DEV), torch.empty(T, H, device=DEV)
        planes = torch.stack([src * 0.25, src * 0.75])        # two pieces of a split product
        K().state_space_operands(planes, 2, row, w, b, dtb, rate, carried, ctx, q, k, u, step, la, H, G, d, dv)
        o = 0
        for s, n in cut:
            got[s].append([t[o:o + n] for t in (q, k, u, step, la)])
            o += n
            at[s] += n
    tol = 1e-5 if dtype == "float32" else KTOL[dtype]
    for s in x:
        z = x[s][:at[s]]
        y = plain.silu(plain.causal_conv(z[:, inner:inner + C], f64(w), f64(b)))
        sz = plain.softplus(z[:, inner + C:inner + C + H] + f64(dtb))
        q, k, u, step, la = (torch.cat([g[i] for g in got[s]]) for i in range(5))
        n = at[s]
        for t, heads, size, ref in ((u, H, dv, y[:, :inner]), (k, G, d, y[:, inner:inner + G * d]), (q, G, d, y[:, inner + G * d:])):
            t = t.view(n, heads, -1)
            assert rel(t[..., :size].reshape(n, -1), ref) < tol and not bool(t[..., size:].any())
        assert rel(step, sz) < 1e-5 and rel(la, -f64(rate) * sz) < 1e-5
        if taps > 1:
            last = np.concatenate([np.zeros((taps - 1, C)), z[:, inner:inner + C]])[-(taps - 1):]
            assert rel(carried[s], last) < 1e-6
    K().check_device_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("geom", [(5, 24, 15, 8), (4, 64, 128, 32), (1, 6, 10, 2), (2, 256, 48, 256), (3, 10, 7, 0), (2, 20, 8, 20)])
def test_rotated_heads_are_the_recurrences_operands(dtype, geom):
    """Partial and whole rotation (dimension i with i + n/2), none at all, the factor on the keys after it, values as they are."""
    H, d, dv, nrot = geom
    dt, r, T = DT[dtype], rng(sum(geom)), 13
    row = (H * (2 * d + dv) + 7) // 8 * 8 + 8
    src = dev(r.standard_normal((T, row)))
    pos = r.integers(0, 5000, T)
    cs = None
    if nrot:
        from hfcpu_b200.parts.rotary import Rotary
        rot = Rotary(d, nrot, 700.0)
        rot.prepare(5000, torch.device(DEV))
        cs = rot.cos_sin
    q, k = (torch.full((T, H * K().padded_head(d)), 3.0, dtype=dt, device=DEV) for _ in range(2))
    u = torch.full((T, H * K().padded_head(dv)), 3.0, dtype=dt, device=DEV)
    K().rotate_heads(torch.stack([src * 0.5] * 2), 2, row, cs, nrot, torch.tensor(pos, dtype=torch.int32, device=DEV), 0.3, q, k, u, H, d, dv)
    x = f64(src)
    turn = lambda a: plain.rotate_half_layout(a, pos, {"dims": nrot, "base": 700.0}) if nrot else a
    tol = 1e-5 if dtype == "float32" else KTOL[dtype]
    for t, n, ref in ((q, d, turn(x[:, :H * d].reshape(T, H, d))), (k, d, 0.3 * turn(x[:, H * d:2 * H * d].reshape(T, H, d))),
                      (u, dv, x[:, 2 * H * d:2 * H * d + H * dv].reshape(T, H, dv))):
        t = t.view(T, H, -1)
        assert rel(t[..., :n], ref) < tol and not bool(t[..., n:].any())
    K().check_device_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("C,parts", [(120, 2), (51, 3), (512, 1), (192, 4), (640, 5), (4096, 1), (6000, 1), (8192, 2), (11, 1), (75, 5), (300, 2)])
@pytest.mark.parametrize("gate_first", [True, False])
def test_norm_in_parts_and_gate(dtype, C, parts, gate_first):
    """The gate before the norm (then a weight) and behind it, into a column slice of a wider array."""
    dt, r, T, eps = DT[dtype], rng(C + parts), 7, 1e-4
    o, g = dev(r.standard_normal((T, C))), dev(2 * r.standard_normal((3, T, C + 12)))
    w = dev(r.uniform(0.5, 1.5, C)) if gate_first else None
    wide = torch.full((T, C + 24), 5.0, dtype=dt, device=DEV)
    K().part_norm_gate(o, parts, eps, g, 3, C + 12, 4, w, gate_first, wide[:, 8:8 + C])
    gate = plain.silu(f64(g).sum(0)[:, 4:4 + C])
    if gate_first:
        want = plain.rms_norm_parts(f64(o) * gate, f64(w), parts, eps)
    else:
        want = plain.unit_rms(f64(o).reshape(T, parts, -1), eps).reshape(T, C) * gate
    assert rel(wide[:, 8:8 + C], want) < (1e-5 if dtype == "float32" else KTOL[dtype])
    assert bool((wide[:, :8] == 5.0).all()) and bool((wide[:, 8 + C:] == 5.0).all())
    K().check_device_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("geom", [(6, 3, 24, 40, 72), (8, 2, 64, 64, 256), (4, 1, 128, 128, 256), (2, 1, 20, 12, 44), (3, 3, 7, 5, 36), (32, 8, 128, 128, 512)])
@pytest.mark.parametrize("T", [3, 200])
def test_norm_over_the_whole_projection(dtype, geom, T):
    """Queries and keys normed over all heads at once, values as they are, sigmoid gates; keys and values to scattered slots;
    and the same rows without keys and values of their own."""
    H, G, d, dv, E = geom
    dt, r, eps = DT[dtype], rng(sum(geom) + T), 1e-3
    n_rows = H * d + G * (d + dv) + H
    from hfcpu_b200.weights.loader import pad_rows
    a, w = dev(r.standard_normal((T, E)), dt), pad_rows(dev(0.2 * r.standard_normal((n_rows, E)), dt))
    qw, kw = dev(r.uniform(0.5, 1.5, H * d)), dev(r.uniform(0.5, 1.5, G * d))
    pages, bs = T // 8 + 2, 8
    kc, vc = torch.zeros(pages, bs, G, d, dtype=dt, device=DEV), torch.zeros(pages, bs, G, dv, dtype=dt, device=DEV)
    slots = torch.tensor(r.permutation(pages * bs)[:T], dtype=torch.int32, device=DEV)
    q, gates = torch.empty(T, H * d, dtype=dt, device=DEV), torch.empty(T, H, device=DEV)
    buf = torch.empty(T, w.shape[0], device=DEV)
    K().linear_row_norm_kv(a, w, buf, qw, kw, eps, slots, q, kc, vc, gates, H, G, d, dv)
    z = f64(a) @ f64(w).T
    QD, KD, VD = H * d, G * d, G * dv
    tol = 1e-5 if dtype == "float32" else KTOL[dtype]
    s = slots.long()
    assert rel(q, plain.rms_norm(z[:, :QD], f64(qw), eps)) < tol
    assert rel(kc.view(-1, KD)[s], plain.rms_norm(z[:, QD:QD + KD], f64(kw), eps)) < tol
    assert rel(vc.view(-1, VD)[s], z[:, QD + KD:QD + KD + VD]) < tol
    assert rel(gates, plain.sigmoid(z[:, QD + KD + VD:QD + KD + VD + H])) < (1e-5 if dtype == "float32" else 2e-5)
    rest = [i for i in range(pages * bs) if i not in set(slots.tolist())]
    assert not bool(kc.view(-1, KD)[rest].any()) and not bool(vc.view(-1, VD)[rest].any())
    w2 = pad_rows(torch.cat([w[:QD], w[QD + KD + VD:QD + KD + VD + H]]))
    q2, gates2 = torch.empty_like(q), torch.empty_like(gates)
    K().linear_row_norm_kv(a, w2, torch.empty(T, w2.shape[0], device=DEV), qw, None, eps, None, q2, kc, vc, gates2, H, 0, d, dv)
    assert rel(q2, plain.rms_norm(z[:, :QD], f64(qw), eps)) < tol and rel(gates2, f64(gates)) < 2e-5
    att_rows = dev(r.standard_normal((T, H * dv)), dt)
    wide = torch.full((T, H * dv + 16), 5.0, dtype=dt, device=DEV)
    K().head_gate(att_rows, gates, wide[:, 8:8 + H * dv], H, dv)
    assert rel(wide[:, 8:8 + H * dv], (f64(att_rows).reshape(T, H, dv) * f64(gates)[:, :, None]).reshape(T, -1)) < tol
    assert bool((wide[:, :8] == 5.0).all()) and bool((wide[:, 8 + H * dv:] == 5.0).all())
    K().check_device_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [(5, 72, 100), (130, 256, 512), (1, 44, 24), (300, 328, 392), (300, 256, 100), (40, 128, 36)])
def test_clamped_gate_with_biases(dtype, shape):
    """Values far beyond the limit on both sides, so that every clamp is at work; the plain sum and the column-slice form."""
    from hfcpu_b200.config import PartSpec
    from hfcpu_b200.parts import make_part
    T, width, ff = shape
    r, dt = rng(sum(shape)), DT[dtype]
    part = make_part("ffn", PartSpec("gated", {"hidden_size": width, "intermediate_size": ff, "prefix": "m", "activation": "clamped",
                                               "clamp": {"limit": 0.9, "alpha": 1.702, "offset": 1.0}, "bias_suffix": ".b",
                                               "names": {"gate": "gate", "up": "up", "down": "down"}}))
    tensors = {s.name: dev((1.0 if s.name.endswith(".b") else 0.2) * r.standard_normal(s.shape), dt) for s in part.tensor_specs()}
    part.bind(tensors, dt, torch.device(DEV))
    W = {k: f64(v) for k, v in tensors.items()}
    ctx = step_ctx([(0, T)], dt)
    xn, res = dev(r.standard_normal((T, width)), dt), dev(r.standard_normal((T, width)))
    g, u = f64(xn) @ W["m.gate"].T + W["m.gate.b"], f64(xn) @ W["m.up"].T + W["m.up.b"]
    assert g.max() > 2 and u.max() > 2 and u.min() < -2
    out = res.clone()
    part.forward(ctx, xn, out)
    assert rel(out, f64(res) + plain.clamped_ff({"limit": 0.9}, W, "m", f64(xn))) < (2e-5 if dtype == "float32" else 2e-2)
    wide = torch.full((T, ff + 24), 5.0, dtype=dt, device=DEV)
    part.operand(ctx, xn, wide[:, 16:16 + ff])
    gc, uc = np.minimum(g, 0.9), np.clip(u, -0.9, 0.9)
    assert rel(wide[:, 16:16 + ff], gc * plain.sigmoid(1.702 * gc) * (uc + 1)) < (1e-5 if dtype == "float32" else KTOL[dtype])
    assert bool((wide[:, :16] == 5.0).all()) and bool((wide[:, 16 + ff:] == 5.0).all())
    K().check_device_errors()


def test_logit_cap():
    r = rng(0)
    x = dev(40 * r.standard_normal((5, 333)))
    want = plain.soft_cap(f64(x), 12.5)
    K().softcap_(x, 12.5)
    assert rel(x, want) < 1e-6 and float(x.abs().max()) <= 12.5


MIXERS = {
    "mamba2": (m2(6, 20, 24, 3, 4, 2), plain.mamba2), "mamba2_tiles": (m2(4, 64, 128, 1, 4, 1), plain.mamba2),
    "mamba2_one_tap": (m2(2, 11, 7, 2, 1, 1), plain.mamba2), "retention": (ret(24, 15, (0.9, 0.999, 0.5), 8, 500.0), plain.retention),
    "retention_tiles": (ret(128, 128, (0.97, 0.9999), 128, 10000.0), plain.retention),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", list(MIXERS))
def test_recurrent_mixer_whole_against_cut(dtype, which):
    """The mixer part on one request whole, and on the same request in portions (two tokens, a chunk's edge) beside another
    request's single tokens."""
    from hfcpu_b200.config import config_from_dict
    from hfcpu_b200.parts import make_part
    spec, oracle = MIXERS[which]
    E, eps, dt, r = 136, 1e-5, DT[dtype], rng(len(which))
    plan = config_from_dict(model(50, E, eps, 0.0, [layer(spec, None)])).plan()
    positions = {n: make_part("position", p) for n, p in plan.positions.items()}
    for p in positions.values():
        p.prepare(512, torch.device(DEV))
    part = make_part("mixer", plan.layers[0].mixer, positions=positions)
    tensors = {s.name: dev(0.3 * r.standard_normal(s.shape) + (1.0 if s.name.endswith(("norm", ".D")) else 0.0), dt) for s in part.tensor_specs()}
    part.bind(tensors, dt, torch.device(DEV))
    Wd = {k: f64(v) for k, v in tensors.items()}
    n = 240
    h = {s: dev(r.standard_normal((n, E)), dt) for s in (0, 1)}
    want = {s: oracle(spec["mixer"], Wd, "l0.mix", f64(h[s]), eps) for s in h}
    runs = {"whole": [[(0, 0, n)], [(1, 0, n)]], "cut": []}
    at = {0: 0, 1: 0}
    for k, size in enumerate([1, 63, 2, 65, 1, 3, 64, 15, 26]):
        cut = [(0, at[0], at[0] + size)] + ([(1, at[1], at[1] + 1)] if k else [])
        runs["cut"].append(cut)
        for s, _, b in cut:
            at[s] = b
    assert at[0] == n
    for cuts in runs.values():
        state = torch.zeros(2, *part.state_spec().shape, dtype=torch.float32, device=DEV)
        got = {0: [], 1: []}
        for cut in cuts:
            ctx = step_ctx([(s, b - a) for s, a, b in cut], dt, np.concatenate([np.arange(a, b) for _, a, b in cut]))
            xn = torch.cat([h[s][a:b] for s, a, b in cut])
            y = torch.zeros(xn.shape[0], E, dtype=torch.float32, device=DEV)
            part.forward(ctx, xn, y, None, state, True)
            o = 0
            for s, a, b in cut:
                got[s].append(y[o:o + b - a].clone())
                o += b - a
        for s in got:
            rows = torch.cat(got[s])
            assert rel(rows, want[s][:rows.shape[0]]) < (5e-5 if dtype == "float32" else 2e-2), s
    K().check_device_errors()


# ---- the engine -------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for i, (n, c) in enumerate(CONFIGS.items()):
        out[n] = make_folder(c, str(tmp_path_factory.mktemp(f"tupalorn_{n}")), 31 + i)
        out[n + "16"] = make_folder(c, str(tmp_path_factory.mktemp(f"tupalorn_{n}16")), 31 + i, torch.bfloat16)
    return out


LENGTHS = {"odd": [1, 19, 70, 130, 33], "wide": [3, 150, 64, 129, 260], "thin": [2, 9, 41]}
FAMILIES = {"whole": traces.whole, "tail": traces.tail_one_by_one, "portions": traces.portions, "mixed": traces.mixed}


def assert_rows(got, ref, tol, what="the plain implementation"):
    keys = sorted(got, key=lambda k: (str(k[0]), k[1]))
    errs = [float((got[k].double() - ref[k[0]][k[1]].double()).abs().max() / ref[k[0]][k[1]].double().abs().max()) for k in keys]
    over = [(k, e) for k, e in zip(keys, errs) if e > tol]
    assert not over, (f"{len(over)} of {len(keys)} rows differ from {what}; first: request {over[0][0][0]} position {over[0][0][1]} "
                      f"(error {over[0][1]:.3g})")


def engine_for(folder, block, dtype, max_tokens, max_requests=4):
    import hfcpu_b200
    m = hfcpu_b200.load_model(folder, DT[dtype], DEV)
    return hfcpu_b200.Engine(m, block_size=block, max_tokens=max_tokens, max_requests=max_requests, ctx_max=4096)


def check_clean(eng):
    K().check_device_errors()
    eng.cache.check()
    assert eng.cache.pages_in_use() == 0 and eng.slots.free_count == eng.max_requests


_WHOLE = {}


@pytest.mark.parametrize("family", list(FAMILIES))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_cuttings_match_plain(folders, name, dtype, family):
    """Whole prompts, a tail decoded token by token, portions down to two tokens, and mixed batches of up to four requests
    in a pool sized for the peak, so that pages and slots are used again."""
    folder = folders[name if dtype == "float32" else name + "16"]
    reqs = requests(CONFIGS[name]["vocab"], LENGTHS[name], seed=3)
    steps = FAMILIES[family](reqs)
    eng = engine_for(folder, BLOCKS[name], dtype, traces.peak_tokens(steps, round_to=BLOCKS[name]))
    got = traces.run_in_process(eng, steps, check=eng.cache.check)
    check_clean(eng)
    ref = {r: plain_logits(folder, ids) for r, ids in reqs.items()}
    assert len(got) == sum(len(v) for v in reqs.values())
    assert_rows(got, ref, TOL[dtype])
    if family == "whole":
        _WHOLE[(name, dtype)] = got
    elif (name, dtype) in _WHOLE:
        base = _WHOLE[(name, dtype)]
        assert_rows(got, {r: torch.stack([base[(r, p)] for p in range(len(ids))]) for r, ids in reqs.items()}, SELF_TOL[dtype],
                    "the whole-prompt run")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["odd", "wide"])
def test_long_decoding(folders, name, dtype):
    """Every token a step of its own (from the second bfloat16 step on a replayed graph, mixer and feed-forward on two of its
    branches), two requests side by side, past several pages, windows and chunks."""
    folder = folders[name if dtype == "float32" else name + "16"]
    reqs = requests(CONFIGS[name]["vocab"], [230, 75], seed=8)
    n = max(len(v) for v in reqs.values())
    steps = []
    for p in range(n):
        entries = [{"id": r, "tokens": [ids[p]], "want": [0], "_pos": p} for r, ids in reqs.items() if p < len(ids)]
        steps.append({"step": p, "entries": entries, "end": [r for r, ids in reqs.items() if p == len(ids) - 1]})
    eng = engine_for(folder, BLOCKS[name], dtype, 384)
    got = traces.run_in_process(eng, steps)
    check_clean(eng)
    assert_rows(got, {r: plain_logits(folder, ids) for r, ids in reqs.items()}, TOL[dtype])


def last_rows(folder, dtype, ids, tails, block=8, size=512):
    """The last position's logits with the last ``tail`` tokens as a portion (1: as a single token) behind the rest."""
    import hfcpu_b200
    eng = engine_for(folder, block, dtype, size, max_requests=1)
    out = []
    for tail in tails:
        eng.add_request("a")
        eng.step([hfcpu_b200.StepEntry("a", ids[:len(ids) - tail], [])])
        out.append(eng.step([hfcpu_b200.StepEntry("a", ids[len(ids) - tail:], [tail - 1])])[0].float().cpu().clone())
        eng.finish_request("a")
    K().check_device_errors()
    return out


# Models from whose last position exactly the last `reach` tokens are seen (a layer's own window; or, where the second layer
# reads the first one's keys, the wider of the two, since a layer's output enters the next layer's queries only).
WINDOWS = {
    "plain": (20, lambda: [layer(att(4, 2, 16, 24, 0.5, 20), 48)]),
    "tiled": (40, lambda: [layer(att(4, 2, 64, 64, 0.3, 40), 48)]),
    "reader_sees_further": (37, lambda: [layer(att(4, 2, 64, 64, 0.3, 9), 48), layer(att(4, 2, 64, 64, 0.3, 37, kv_from=0), 48)]),
    "reader_sees_less_far": (33, lambda: [layer(att(4, 2, 16, 24, 0.5, 33), None), layer(att(4, 2, 16, 24, 0.5, 6, kv_from=0), 48)]),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", list(WINDOWS))
def test_a_changed_token_shows_exactly_inside_the_window(tmp_path, which, dtype):
    """One token is changed at places around the window's far edge: inside, the logits must move and be the plain
    implementation's; outside they must not move at all.  The last tokens come as a portion and as single tokens."""
    reach, layers = WINDOWS[which]
    folder = make_folder(model(150, 64, 1e-5, 30.0, layers()), str(tmp_path / which), 21, DT[dtype])
    n = 3 * reach + 5
    base = requests(150, [n], seed=2)["r0"]
    rows = last_rows(folder, dtype, base, (1, 7))
    for place in (n - 1 - reach - 1, n - 1 - reach, n - reach, n - reach + 1, n - 2):
        ids = list(base)
        ids[place] = (ids[place] + 71) % 150
        want = plain_logits(folder, ids)[n - 1]
        for before, after in zip(rows, last_rows(folder, dtype, ids, (1, 7))):
            assert float((after.double() - want).abs().max() / want.abs().max()) < TOL[dtype], place
            moved = float((after - before).abs().max())
            assert moved > 1e-3 if place >= n - reach else moved == 0.0, (place, moved)


def far_folder(spec, folder, dtype, n, place, far, last):
    """A one-layer model in which what token ``far`` at position ``place`` writes into the state is what the query of token
    ``last`` at position n - 1 reads, whatever lies between.  Retention: per head, the direction that the key projection
    carries onto the last query turned back by the distance; Mamba-2: per head, the direction of the step size.  The far
    token's embedding is the sum of the heads' directions, and every other token's has no part along any of them."""
    cfg = model(150, 64, 1e-5, 60.0, [layer(spec, 48)])

    def edit(t):
        W = {k: v.double().numpy() for k, v in t.items()}
        m = spec["mixer"]
        if spec["type"] == "retention":
            H, d = m["heads"], m["dim"]
            h_last = plain.layer_norm(W["embed"][last][None], W["l0.norm1"], 1e-5)
            q = plain.rotate_half_layout((h_last @ W["l0.mix.q"].T).reshape(1, H, d), [n - 1 - place], m["rot"])[0]
            Wk, n_rot = W["l0.mix.k"].reshape(H, d, -1), m["rot"]["dims"]
            dirs = np.einsum("hd,hde->he", q, Wk)
            # the rotated rows meet the query at another angle from every place: no other token has a part along them either
            off = np.concatenate([np.einsum("hd,hde->he", q[:, n_rot:], Wk[:, n_rot:]), Wk[:, :n_rot].reshape(H * n_rot, -1)])
        else:
            t["l0.mix.A_log"].fill_(-8.0)
            t["l0.mix.dt_bias"].fill_(-7.0)
            t["l0.mix.in"][-m["heads"]:] *= 3
            off = dirs = W["l0.mix.in"][-m["heads"]:]
        dirs, off = dirs * W["l0.norm1"], off * W["l0.norm1"]
        off -= off.mean(-1, keepdims=True)                    # (the norm takes the mean off)
        dirs /= np.linalg.norm(dirs, axis=-1, keepdims=True)
        basis = np.linalg.qr(off.T)[0]
        e = W["embed"].copy()
        e -= (e @ basis) @ basis.T
        e[far], e[last] = 4 * dirs.sum(0), W["embed"][last]
        t["embed"].copy_(torch.from_numpy(e))
    return make_folder(cfg, folder, 23, dtype, edit=edit)


FAR = {"retention": lambda: ret(24, 20, (0.9997, 0.99995), 4, 100.0), "retention_tiles": lambda: ret(64, 128, (0.9997, 0.9999), 4, 100.0),
       "mamba2": lambda: m2(2, 24, 20, 1, 4, 1)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", list(FAR))
def test_a_far_key_is_found_in_the_state(tmp_path, which, dtype):
    """Hundreds of tokens and one that stands out, far back, on both sides of chunks' edges and right at the start: the last
    position's logits must be the plain implementation's, in which that token decides (taking it away moves them by a large
    part of their size).  The last tokens come as a portion and as a single token."""
    n = 420
    base = [t % 147 for t in requests(150, [n], seed=6)["r0"]]
    for place in (0, 1, 63, 64, 65, 255, 300):
        folder = far_folder(FAR[which](), str(tmp_path / f"{which}_{place}"), DT[dtype], n, place, 149, 148)
        ids = list(base)
        ids[place], ids[n - 1] = 149, 148
        want = plain_logits(folder, ids)[n - 1]
        without = list(ids)
        without[place] = 147
        assert float((plain_logits(folder, without)[n - 1] - want).abs().max()) > 0.25 * float(want.abs().max()), place
        # (bfloat16: one token's key and value make the whole output here, so their rounding does not average out: the stand-in
        # kernels, which round at the same places and nowhere else, are off by 0.033 of the largest logit)
        for row in last_rows(folder, dtype, ids, (1, 5, 70), block=16):
            assert float((row.double() - want).abs().max() / want.abs().max()) < (TOL[dtype] if dtype == "float32" else 5e-2), place


def test_greedy_generation_through_the_entry_point(folders):
    import hfcpu_b200
    for name in ("odd", "wide"):
        folder = folders[name]
        sess = hfcpu_b200.Session(folder, dtype="float32", kv_block=BLOCKS[name], kv_pages=96, max_seqs=4,
                                  max_batched_tokens=48, batch=32, ctx_max=512)
        prompts = list(requests(CONFIGS[name]["vocab"], [7, 33, 1, 60], seed=2).values())
        out = sess.generate(prompts, temp=0, max_tokens=10)
        cfg, W = plain.read_folder(folder)
        for p, comps in zip(prompts, out):
            assert comps[0].tokens == plain.greedy(cfg, W, p, 10)
        assert sess.engine.cache.pages_in_use() == 0


def test_bfloat16_generation_replays_graphs(folders):
    """Steady decoding in bfloat16 goes through captured graphs (the states included) and repeats itself; more requests than
    slots, so that slots are used again; and the graph's two branches give what one after the other gives."""
    import hfcpu_b200
    sess = hfcpu_b200.Session(folders["wide16"], dtype="bfloat16", kv_block=16, kv_pages=128, max_seqs=2, ctx_max=512)
    prompts = list(requests(1032, [19, 130, 64, 5], seed=2).values())
    a = sess.generate(prompts, temp=0, max_tokens=24)
    assert sess.engine.use_graphs and any(s[0] == "ready" for s in sess.engine._graphs.values())
    b = sess.generate(prompts, temp=0, max_tokens=24)
    assert [c[0].tokens for c in a] == [c[0].tokens for c in b] and all(len(c[0].tokens) == 24 for c in a)
    backend = K().backend()
    backend.branches = False
    try:
        other = hfcpu_b200.Session(folders["wide16"], dtype="bfloat16", kv_block=16, kv_pages=128, max_seqs=2, ctx_max=512)
        assert [c[0].tokens for c in other.generate(prompts, temp=0, max_tokens=24)] == [c[0].tokens for c in a]
    finally:
        backend.branches = True
    # and they are the tokens of the plain implementation's first steps where it has a clear winner
    cfg, W = plain.read_folder(folders["wide16"])
    for got, p in zip(a, prompts):
        row = np.sort(plain.forward(cfg, W, p)[-1])
        if row[-1] - row[-2] > 0.5:
            assert got[0].tokens[0] == int(np.argmax(plain.forward(cfg, W, p)[-1]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_program(folders, tmp_path, dtype):
    folder = folders["odd" if dtype == "float32" else "odd16"]
    reqs = requests(211, [1, 19, 70, 33, 50], seed=5)
    steps = traces.mixed(reqs)
    got = traces.run_trace_program(folder, dtype, steps, str(tmp_path), traces.peak_tokens(steps), 211, block_size=8)
    assert_rows(got, {r: plain_logits(folder, ids) for r, ids in reqs.items()}, TOL[dtype])


def test_command_line_generates(folders):
    import subprocess
    import sys
    from conftest import ROOT
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "hfb200"), "--model", folders["wide16"], "--op", "generate",
                        "--stdin-mode", "none", "--prompt-ids", "5,17,3,900", "--temp", "0", "--max-tokens", "6", "--ctx-max", "256",
                        "--kv-pages", "32"],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert "stop=length" in r.stdout or "length" in r.stdout
