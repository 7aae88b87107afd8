"""Tupalorn on a machine without a GPU: configuration and plan, tensor names, what is decided on the host (the window a
shared cache keeps, the chunks of a step, the joined output product), and the engine's host side (batching, states of the
recurrences and of the convolution carried from step to step, shared caches) with the torch stand-in for the CUDA library
against the plain implementation."""
import copy

import numpy as np
import pytest
import torch

import plain_tupalorn as plain
import traces
from tupalorn_util import BLOCKS, CONFIGS, att, layer, m2, make_folder, model, plain_logits, requests, ret


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {n: make_folder(c, str(tmp_path_factory.mktemp(f"tupalorn_{n}")), 31 + i) for i, (n, c) in enumerate(CONFIGS.items())}


def test_plan_follows_the_layer_list():
    from hfcpu_b200.config import TupalornConfig, config_from_dict
    cfg = config_from_dict(CONFIGS["odd"])
    assert isinstance(cfg, TupalornConfig)
    plan = cfg.plan()
    assert [l.mixer.kind for l in plan.layers] == ["mamba2", "paged_attention", "retention", "paged_attention", "paged_attention", "mamba2",
                                                   "paged_attention"]
    assert [(e.layer, e.cache_of) for e in plan.schedule] == [(0, None), (1, None), (2, None), (3, 1), (4, None), (5, None), (6, 1)]
    assert [l.ffn is None for l in plan.layers] == [False, False, True, False, False, False, True]
    assert all(l.norm2 is None and l.block.kind == "parallel_residual" and l.norm1.kind == "layernorm" for l in plan.layers)
    assert plan.layers[0].ffn.args["clamp"] == {"limit": 1.5, "alpha": 1.702, "offset": 1.0}
    # layer 1's cache keeps what layer 3 sees, which is more than it sees itself; the others' own windows
    assert [plan.layers[i].mixer.args["window"] for i in (1, 3, 4, 6)] == [12, 29, 1, 5]
    assert [plan.layers[i].mixer.args["cache_window"] for i in (1, 4)] == [29, 1]
    assert [plan.layers[i].mixer.args["own_kv"] for i in (1, 3, 4, 6)] == [True, False, True, False]
    assert plan.head.args["tensor"] == plan.embedding.args["tensor"] == "embed" and plan.head.args["softcap"] == 20.0
    assert plan.layers[2].mixer.args["decay"] == [0.9, 0.97, 0.995, 0.5, 0.999] and len(plan.positions) == 1
    again = config_from_dict(cfg.to_dict())
    assert again.to_dict() == cfg.to_dict()
    assert config_from_dict(CONFIGS["thin"]).plan().layers[4].mixer.args["position"] is None       # rot.dims 0: no rotation


def test_optional_keys_have_defaults():
    from hfcpu_b200.config import config_from_dict
    d = {"architecture": "Tupalorn", "vocab": 50, "width": 16, "norm": {"eps": 1e-6}, "layers": [
        {"type": "attention", "mixer": {"heads": 2, "dim": 8, "scale": 0.3}, "mlp": None},
        {"type": "mamba2", "mixer": {"heads": 2, "vdim": 8, "state": 4, "conv": 2}},
        {"type": "retention", "mixer": {"heads": 1, "dim": 8, "decay": [0.5]}},
        {"type": "attention", "mixer": {"heads": 2, "dim": 8, "scale": 0.3, "mask": {"size": 7}, "kv_from": 0}}]}
    plan = config_from_dict(d).plan()
    a = plan.layers[0].mixer.args
    assert (a["num_kv_heads"], a["v_head_dim"], a["window"], a["cache_window"]) == (2, 8, 0, 0)
    assert plan.layers[1].mixer.args["groups"] == 1 and plan.layers[1].mixer.args["norm_groups"] == 1
    assert plan.layers[2].mixer.args["v_head_dim"] == 8 and plan.layers[2].mixer.args["position"] is None
    assert plan.head.args["softcap"] == 0.0 and plan.layers[3].mixer.args["window"] == 7


@pytest.mark.parametrize("edit,match", [
    (lambda L: L[0].update(type="convolution"), "convolution"),
    (lambda L: L[0]["mixer"].update(groups=4), "groups"),
    (lambda L: L[0]["mixer"].update(norm_groups=7), "norm groups"),
    (lambda L: L[0]["mixer"].pop("state"), "state"),
    (lambda L: L[2]["mixer"].update(decay=[0.5]), "decay"),
    (lambda L: L[2]["mixer"].update(decay=[0.5, 0.5, 0.5, 0.5, 1.5]), "decay"),
    (lambda L: L[2]["mixer"]["rot"].update(dims=26), "rot.dims"),
    (lambda L: L[3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda L: L[6]["mixer"].update(kv_from=3), "kv_from"),
    (lambda L: L[6]["mixer"].update(kv_from=2), "kv_from"),
    (lambda L: L[6]["mixer"].update(vdim=24), "other sizes"),
    (lambda L: L[4]["mixer"].update(kv_heads=3), "geometry"),
    (lambda L: L[0]["mlp"].update(kind="moe"), "moe"),
    (lambda L: L[0]["mlp"].pop("limit"), "limit"),
])
def test_configuration_errors(edit, match):
    from hfcpu_b200.config import ConfigError, config_from_dict
    bad = copy.deepcopy(CONFIGS["odd"])
    edit(bad["layers"])
    with pytest.raises(ConfigError, match=match):
        config_from_dict(bad)


def test_tensor_names():
    from hfcpu_b200.config import config_from_dict
    from hfcpu_b200.models import build_model_specs
    specs = {s.name: s.shape for s in build_model_specs(config_from_dict(CONFIGS["odd"]))}
    assert specs["embed"] == (211, 72) and specs["final.norm"] == (72,) and "head" not in specs and "l0.norm2" not in specs
    assert specs["l0.mix.in"] == (2 * 120 + 2 * 72 + 6, 72) and specs["l0.mix.conv"] == (264, 4) and specs["l0.mix.conv.b"] == (264,)
    assert specs["l0.mix.dt_bias"] == specs["l0.mix.A_log"] == specs["l0.mix.D"] == (6,)
    assert specs["l0.mix.norm"] == (120,) and specs["l0.mix.o"] == (72, 120)
    assert specs["l0.mlp.gate"] == (100, 72) and specs["l0.mlp.gate.b"] == specs["l0.mlp.up.b"] == (100,) and specs["l0.mlp.down.b"] == (72,)
    assert specs["l1.mix.q"] == (144, 72) and specs["l1.mix.k"] == (72, 72) and specs["l1.mix.v"] == (120, 72) and specs["l1.mix.o"] == (72, 240)
    assert specs["l1.mix.q.norm"] == (144,) and specs["l1.mix.k.norm"] == (72,) and specs["l1.mix.g"] == (6, 72)
    assert specs["l2.mix.q"] == (120, 72) and specs["l2.mix.v"] == specs["l2.mix.g"] == (75, 72) and specs["l2.mix.o"] == (72, 75)
    assert sorted(n for n in specs if n.startswith("l3.mix")) == ["l3.mix.g", "l3.mix.o", "l3.mix.q", "l3.mix.q.norm"]
    assert not any(n.startswith("l2.mlp") for n in specs)


def test_chunks_of_a_step():
    from hfcpu_b200.kernels import DECAY_CHUNK as C
    from hfcpu_b200.kernels import decay_chunk_arrays
    assert decay_chunk_arrays([1, 1, 1]) == {} and decay_chunk_arrays([15, 2]) == {}
    a = decay_chunk_arrays([1, C, 2 * C + 1, 16])
    assert a["t0"].tolist() == [0, 1, C + 1, 2 * C + 1, 3 * C + 1, 3 * C + 2]
    assert a["n"].tolist() == [1, C, C, C, 1, 16] and a["first"].tolist() == [0, 1, 2, 5, 6]


def test_output_products_are_joined_where_the_sizes_allow(folders, tmp_path):
    import hfcpu_b200
    m = hfcpu_b200.load_model(folders["odd"], torch.float32, "cpu")
    assert [l.block.widths for l in m.layers] == [(120, 100), (240, 64), None, (240, 48), (64, 56), (51, 40), None]
    l0 = m.layers[0]
    assert torch.equal(l0.block.w_out, torch.cat([l0.mixer.w_o, l0.ffn.w_down], 1)) and l0.block.b_out is l0.ffn.b_down
    soft = make_folder(CONFIGS["odd"], str(tmp_path), 31, torch.bfloat16)
    m = hfcpu_b200.load_model(soft, torch.bfloat16, "cpu")                  # 16-byte rows only, for the tensor-core product
    assert [l.block.widths for l in m.layers] == [None, (240, 64), None, (240, 48), (64, 56), None, None]


def test_the_shared_cache_keeps_the_widest_readers_window(folders, emu):
    """Layer 1 sees 12 positions, layer 3 reads its cache 29 back: pages behind 12 must not go back to the pool early."""
    import hfcpu_b200
    m = hfcpu_b200.load_model(folders["odd"], torch.float32, "cpu")
    assert m.layers[1].mixer.cache_spec().window == 29 and m.layers[1].mixer.window == 12
    eng = hfcpu_b200.Engine(m, block_size=8, max_tokens=128, max_requests=1)
    assert sorted(g.spec.window for g in eng.cache.groups) == [1, 29]


LENGTHS = {"odd": [1, 19, 70, 27], "wide": [3, 70, 20], "thin": [2, 9, 41]}


@pytest.mark.parametrize("family", ["whole", "portions", "mixed"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_engine_host_side_matches_plain(folders, emu, name, family):
    """Every cutting through the engine (pages, slots, states) with the stand-in kernels gives the plain implementation's
    logits."""
    import hfcpu_b200
    reqs = requests(CONFIGS[name]["vocab"], LENGTHS[name], seed=4)
    steps = {"whole": traces.whole, "portions": lambda r: traces.portions(r, sizes=(7, 2, 16, 3, 5, 2, 11)),
             "mixed": lambda r: traces.mixed(r, max_live=3, prefill_sizes=(9, 2, 5, 17))}[family](reqs)
    m = hfcpu_b200.load_model(folders[name], torch.float32, "cpu")
    eng = hfcpu_b200.Engine(m, block_size=BLOCKS[name], max_tokens=traces.peak_tokens(steps, round_to=BLOCKS[name]), max_requests=3)
    got = traces.run_in_process(eng, steps, check=eng.cache.check)
    assert eng.cache.pages_in_use() == 0 and eng.slots.free_count == 3
    for (r, pos), row in got.items():
        want = plain_logits(folders[name], reqs[r])[pos]
        assert float((row.double() - want).abs().max() / want.abs().max()) < 2e-4, (r, pos)


def test_a_slot_taken_over_starts_from_zero(folders, emu):
    """A request that gets the slot of a finished one must not see its states or its convolution's inputs."""
    import hfcpu_b200
    m = hfcpu_b200.load_model(folders["thin"], torch.float32, "cpu")
    eng = hfcpu_b200.Engine(m, block_size=4, max_tokens=64, max_requests=1)
    ids = requests(97, [11, 11], seed=9)
    for r in ("r0", "r1"):
        eng.add_request(r)
        a = eng.step([hfcpu_b200.StepEntry(r, ids[r][:6], [5])])[0].clone()
        b = eng.step([hfcpu_b200.StepEntry(r, ids[r][6:], [4])])[0].clone()
        eng.finish_request(r)
        want = plain_logits(folders["thin"], ids[r])
        assert float((a.double() - want[5]).abs().max()) < 1e-3 and float((b.double() - want[10]).abs().max()) < 1e-3


def test_greedy_decoding_on_the_stand_in(folders, emu):
    """A prompt and then the arg-max token of every step, request after request in the same slot."""
    import hfcpu_b200
    m = hfcpu_b200.load_model(folders["thin"], torch.float32, "cpu")
    eng = hfcpu_b200.Engine(m, block_size=4, max_tokens=96, max_requests=2)
    cfg, W = plain.read_folder(folders["thin"])
    for ids in requests(97, [5, 17], seed=1).values():
        eng.add_request("a")
        out, logits = [], eng.step([hfcpu_b200.StepEntry("a", ids, [len(ids) - 1])])
        for _ in range(6):
            out.append(int(logits[0].argmax()))
            logits = eng.step([hfcpu_b200.StepEntry("a", [out[-1]], [0])])
        eng.finish_request("a")
        assert out == plain.greedy(cfg, W, ids, 6)


# ---- the plain implementation's own pieces ---------------------------------------------------------------------------
def test_plain_recurrence_is_a_weighted_sum():
    """S_t^T q_t unrolled: o_t = sum_(s <= t) (q_t . k_s) (product of a over s+1 .. t) u_s."""
    r = np.random.default_rng(0)
    T, d, dv = 9, 5, 3
    a, k, u, q = r.uniform(0.3, 1, T), r.standard_normal((T, d)), r.standard_normal((T, dv)), r.standard_normal((T, d))
    want = np.stack([sum((q[t] @ k[s]) * np.prod(a[s + 1:t + 1]) * u[s] for s in range(t + 1)) for t in range(T)])
    assert np.allclose(plain.scalar_decay_scan(a, k, u, q), want)


def test_plain_convolution_reads_the_last_taps():
    x = np.arange(12.0).reshape(6, 2)
    w = np.array([[1.0, 10.0, 100.0], [0.0, 0.0, 1.0]])
    y = plain.causal_conv(x, w, np.array([0.5, 0.0]))
    assert y[0, 0] == 0.5 and y[1, 0] == 100 * 2 + 10 * 0 + 0.5 and y[4, 0] == 8 * 100 + 6 * 10 + 4 + 0.5
    assert np.array_equal(y[:, 1], x[:, 1])


def test_the_clamps_and_the_window_matter():
    """With these weights a limit left out, or a window off by one, changes the logits by far more than the tolerance."""
    cfg = model(60, 24, 1e-5, 10.0, [layer(att(2, 1, 8, 8, 0.5, 4), 32, 0.3), layer(m2(2, 8, 4, 1, 3, 2), 16, 0.3),
                                     layer(ret(8, 8, (0.9,), 4, 50.0), 16, 0.3)])
    import tempfile
    with tempfile.TemporaryDirectory() as t:
        c, W = plain.read_folder(make_folder(cfg, t, 3))
    ids = requests(60, [20], seed=3)["r0"]
    base = plain.forward(c, W, ids)
    for edit in (lambda d: d["layers"][0]["mlp"].update(limit=1e9), lambda d: d["layers"][0]["mixer"]["mask"].update(size=5),
                 lambda d: d["layers"][0]["mixer"]["mask"].update(size=3), lambda d: d["layers"][1]["mixer"].update(norm_groups=1),
                 lambda d: d["layers"][2]["mixer"].update(decay=[0.91]), lambda d: d.update(logit_softcap=12.0)):
        d = copy.deepcopy(c)
        edit(d)
        assert np.abs(plain.forward(d, W, ids) - base).max() > 0.01 * np.abs(base).max()


def test_a_model_without_attention_keeps_no_pages(tmp_path, emu):
    """Only recurrent layers: no cache group at all, the requests' lengths still advance the rotation."""
    import hfcpu_b200
    cfg = model(60, 24, 1e-5, 10.0, [layer(ret(8, 8, (0.9, 0.99), 4, 50.0), 16, 0.3), layer(m2(2, 8, 4, 1, 3, 2), 16, 0.3)])
    folder = make_folder(cfg, str(tmp_path), 5)
    reqs = requests(60, [30, 7, 12], seed=3)
    steps = traces.mixed(reqs, max_live=2, prefill_sizes=(5, 2, 9))
    m = hfcpu_b200.load_model(folder, torch.float32, "cpu")
    eng = hfcpu_b200.Engine(m, block_size=8, max_tokens=64, max_requests=2)
    assert eng.cache.groups == []
    got = traces.run_in_process(eng, steps, check=eng.cache.check)
    for (r, pos), row in got.items():
        want = plain_logits(folder, reqs[r])[pos]
        assert float((row.double() - want).abs().max() / want.abs().max()) < 2e-4, (r, pos)
