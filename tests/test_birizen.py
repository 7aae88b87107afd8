"""Birizen on a machine without a GPU: configuration and plan, the run order with its passes, tensor names, and the engine's
host side (batching, states and caches per pass, what is handed over between layers and passes) with the torch stand-in for
the CUDA library against the plain implementation."""
import copy

import numpy as np
import pytest
import torch

import plain_birizen as plain
import traces
from birizen_util import BLOCKS, CONFIGS, far_folder, latent, layer, lightning, make_folder, model, moe, plain_logits, requests


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {n: make_folder(c, str(tmp_path_factory.mktemp(f"birizen_{n}")), 31 + i) for i, (n, c) in enumerate(CONFIGS.items())}


def test_plan_follows_the_layer_list():
    from hfcpu_b200.config import BirizenConfig, config_from_dict
    cfg = config_from_dict(CONFIGS["odd"])
    assert isinstance(cfg, BirizenConfig)
    plan = cfg.plan()
    assert [l.mixer.kind for l in plan.layers] == ["lightning_attention", "latent_attention", "lightning_attention", "latent_attention",
                                                   "lightning_attention"]
    assert [(e.layer, e.enter, e.cache_of) for e in plan.schedule] == [
        (0, None, None), (1, ("loop", 0), None), (2, None, None), (1, ("loop", 1), None), (2, None, None), (3, None, None), (4, None, None)]
    assert plan.transitions["loop"].args["first"] is False and plan.transitions["loop"].args["passes"] == 2
    assert [l.ffn is None for l in plan.layers] == [False, False, True, False, True]
    assert all(l.block.kind == "sandwich_residual" and l.norm1.kind == "rmsnorm" for l in plan.layers)
    f = plan.layers[0].ffn.args
    assert f["clamp"] == {"limit": 0.6, "alpha": 1.702, "offset": 1.0} and f["shared_clamp"]["limit"] == 1.1 and f["groups"] == (3, 2)
    assert f["router"] == "sigmoid" and f["group_best"] == 2 and f["renorm"] and plan.layers[1].ffn.args["groups"] is None
    assert plan.layers[3].ffn.args["shared_size"] == 0 and plan.layers[3].ffn.args["shared_clamp"] is None
    assert plan.layers[0].mixer.args["decay"] == [0.9, 0.98, 0.999, 0.4, 1.0] and plan.layers[0].mixer.args["key_scale"] == 1.0
    assert len(plan.positions) == 2 and plan.head.args["tensor"] == plan.embedding.args["tensor"] == "embed"
    again = config_from_dict(cfg.to_dict())
    assert again.to_dict() == cfg.to_dict()


def test_run_order_at_the_edges():
    from hfcpu_b200.config import config_from_dict
    order = lambda loop: [(e.layer, e.enter and e.enter[1]) for e in config_from_dict(dict(CONFIGS["thin"], loop=dict(zip(
        ("start", "stop", "times"), loop)))).plan().schedule]
    assert order((0, 3, 2)) == [(0, 0), (1, None), (2, None), (0, 1), (1, None), (2, None)]
    assert order((2, 3, 3)) == [(0, None), (1, None), (2, 0), (2, 1), (2, 2)]
    assert order((1, 3, 0)) == [(0, None)] and order((1, 1, 4)) == [(0, None), (1, None), (2, None)]
    plan = config_from_dict(CONFIGS["flat"]).plan()
    assert not plan.transitions and [e.enter for e in plan.schedule] == [None, None]
    assert config_from_dict(CONFIGS["wide"]).plan().transitions["loop"].args["first"] is True


def test_optional_keys_have_defaults():
    from hfcpu_b200.config import config_from_dict
    d = {"architecture": "Birizen", "vocab": 50, "width": 16, "norm": {"eps": 1e-6}, "layers": [
        {"type": "lightning", "mixer": {"heads": 2, "dim": 8, "decay": [0.5, 1]}},
        {"type": "latent_attention", "mixer": {"heads": 2, "dim": 8, "rot_dim": 0, "q_rank": 4, "kv_rank": 4, "scale": 0.3},
         "mlp": {"kind": "moe", "expert": {"ff": 8, "limit": 1.0}, "router": {"experts": 2, "top": 1}}}]}
    plan = config_from_dict(d).plan()
    assert plan.layers[0].mixer.args["v_head_dim"] == plan.layers[1].mixer.args["v_head_dim"] == 8
    assert plan.layers[1].mixer.args["position"] is None and plan.layers[1].ffn.args["shared_size"] == 0 and plan.layers[0].ffn is None


@pytest.mark.parametrize("edit,match", [
    (lambda L: L[0].update(type="retention"), "retention"),
    (lambda L: L[0]["mixer"].update(decay=[0.5]), "decay"),
    (lambda L: L[0]["mixer"].update(decay=[0.5, 0.5, 0.5, 0.5, 1.5]), "decay"),
    (lambda L: L[1]["mixer"].update(rot_dim=9), "rot_dim"),
    (lambda L: L[1]["mixer"]["rot"].update(dims=8), "rot.dims"),
    (lambda L: L[1]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda L: L[1]["mixer"].pop("q_rank"), "q_rank"),
    (lambda L: L[0]["mlp"].update(kind="dense"), "dense"),
    (lambda L: L[0]["mlp"]["router"].update(top=10), "top"),
    (lambda L: L[0]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda L: L[3]["mlp"]["router"]["groups"].update(keep=1), "groups"),
    (lambda L: L[0]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda L: L[0]["mlp"]["shared"].pop("ff"), "ff"),
])
def test_configuration_errors(edit, match):
    from hfcpu_b200.config import ConfigError, config_from_dict
    bad = copy.deepcopy(CONFIGS["odd"])
    edit(bad["layers"])
    with pytest.raises(ConfigError, match=match):
        config_from_dict(bad)
    for loop in ((3, 1, 2), (0, 6, 2), (0, 1, -1)):
        with pytest.raises(ConfigError):
            config_from_dict(dict(CONFIGS["odd"], loop=dict(zip(("start", "stop", "times"), loop))))


def test_tensor_names():
    from hfcpu_b200.config import config_from_dict
    from hfcpu_b200.models import build_model_specs
    all_specs = build_model_specs(config_from_dict(CONFIGS["odd"]))
    specs = {s.name: s.shape for s in all_specs}
    assert specs["embed"] == (211, 72) and specs["final.norm"] == (72,) and "head" not in specs
    assert specs["loop.in"] == (72, 144) and specs["loop.step"] == (2, 72)
    assert specs["l0.mix.q"] == specs["l0.mix.k"] == (100, 72) and specs["l0.mix.v"] == specs["l0.mix.g"] == (75, 72)
    assert specs["l0.mix.norm"] == (75,) and specs["l0.mix.o"] == (72, 75)
    assert specs["l0.mlp.e8.gate"] == specs["l0.mlp.e0.up"] == (40, 72) and specs["l0.mlp.e3.down"] == (72, 40)
    assert specs["l0.mlp.router"] == (9, 72) and specs["l0.mlp.correction"] == (9,)
    assert specs["l0.mlp.shared.gate"] == specs["l0.mlp.shared.up"] == (56, 72) and specs["l0.mlp.shared.down"] == (72, 56)
    assert specs["l1.mix.dq"] == (28, 72) and specs["l1.mix.dq.norm"] == (28,) and specs["l1.mix.uq"] == (6 * 34, 28)
    assert specs["l1.mix.dkv"] == (40, 72) and specs["l1.mix.dkv.norm"] == (30,) and specs["l1.mix.uk"] == (144, 30)
    assert specs["l1.mix.uv"] == (120, 30) and specs["l1.mix.sink"] == (6,) and specs["l1.mix.g"] == (120, 72) and specs["l1.mix.o"] == (72, 120)
    assert all(specs[f"l1.{n}"] == (72,) for n in ("norm1", "norm1b", "norm2", "norm2b"))
    assert not any(n.startswith(("l2.mlp", "l3.mlp.shared")) for n in specs)
    # the norms around a feed-forward that is not there may be stored or not
    assert {s.name for s in all_specs if s.optional} == {"l2.norm2", "l2.norm2b", "l4.norm2", "l4.norm2b"}


def test_unread_norms_may_be_left_out(folders, tmp_path, emu):
    import hfcpu_b200
    from hfcpu_b200.weights import write_safetensors, weights_path
    ids = requests(64, [12], seed=1)["r0"]

    def last(folder):
        eng = hfcpu_b200.Engine(hfcpu_b200.load_model(folder, torch.float32, "cpu"), block_size=8, max_tokens=64, max_requests=1)
        eng.add_request("a")
        return eng.step([hfcpu_b200.StepEntry("a", ids, [11])])[0].clone()
    import shutil
    shutil.copytree(folders["flat"], str(tmp_path / "m"))
    W = {k: torch.from_numpy(v).float() for k, v in plain.read_safetensors(weights_path(folders["flat"])).items()}
    assert W.pop("l0.norm2") is not None and W.pop("l0.norm2b") is not None
    write_safetensors(weights_path(str(tmp_path / "m")), W)
    assert torch.equal(last(folders["flat"]), last(str(tmp_path / "m")))


def test_every_pass_has_a_state_and_a_cache_of_its_own(folders, emu):
    import hfcpu_b200
    m = hfcpu_b200.load_model(folders["odd"], torch.float32, "cpu")
    eng = hfcpu_b200.Engine(m, block_size=8, max_tokens=128, max_requests=2)
    caches = [eng.cache.entry_cache(i) for i in (1, 3, 5)]
    assert len({c.k.data_ptr() for c in caches}) == 3
    states = [eng.slots.entry_state(i) for i in (0, 2, 4, 6)]
    assert len({s.data_ptr() for s in states}) == 4 and all(s.dtype == torch.float32 for s in states)
    assert eng.slots.entry_state(1) is None


LENGTHS = {"odd": [1, 19, 70, 27], "wide": [3, 70, 20], "thin": [2, 9, 41], "flat": [17, 2, 33], "latent": [30, 2, 11]}


@pytest.mark.parametrize("family", ["whole", "portions", "mixed"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_engine_host_side_matches_plain(folders, emu, name, family):
    """Every cutting through the engine (pages, slots, states, passes) with the stand-in kernels gives the plain
    implementation's logits."""
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


def test_a_loop_around_pre_norm_layers(emu):
    """The transition in front of a pass works with another block too: a plan of pre-norm layers with the same step, the
    operand handed over or made by the transition itself."""
    import dataclasses
    from hfcpu_b200 import Engine, StepEntry
    from hfcpu_b200.config import LayerSpec, ModelPlan, PartSpec, ScheduleEntry, config_from_dict
    from hfcpu_b200.models import Model
    from hfcpu_b200.weights import random_tensors
    cfg = config_from_dict(CONFIGS["thin"])
    plan = cfg.plan()
    layers = [LayerSpec(prefix=l.prefix, block=PartSpec("prenorm_residual"), norm1=l.norm1, mixer=l.mixer, norm2=l.norm2, ffn=None)
              for l in plan.layers]
    plan = dataclasses.replace(plan, layers=layers)
    m = Model(cfg, torch.float32, torch.device("cpu"), plan=plan)
    W = random_tensors(m.tensor_specs(), 3, torch.float32, std=0.3)
    m.bind(W)
    eng = Engine(m, block_size=4, max_tokens=32, max_requests=1)
    ids = requests(97, [9], seed=2)["r0"]
    eng.add_request("a")
    got = eng.step([StepEntry("a", ids, list(range(9)))]).double().numpy()
    N = {k: v.double().numpy() for k, v in W.items()}
    x0 = x = N["embed"][ids]
    for i, t in plain.run_order(CONFIGS["thin"]):
        if t is not None:
            x = plain.enter_pass(N, t, x, x0)
        L = CONFIGS["thin"]["layers"][i]
        mixer = {"lightning": plain.lightning, "latent_attention": plain.latent_attention}[L["type"]]
        x = x + mixer(L["mixer"], N, f"l{i}.mix", plain.rms_norm(x, N[f"l{i}.norm1"], 1e-4), 1e-4)
    want = plain.rms_norm(x, N["final.norm"], 1e-4) @ N["embed"].T
    assert np.abs(got - want).max() < 1e-4 * np.abs(want).max()


# ---- the plain implementation's own pieces ---------------------------------------------------------------------------
def test_plain_recurrence_is_a_weighted_sum():
    r = np.random.default_rng(0)
    T, d, dv, a = 9, 5, 3, 0.8
    k, v, q = r.standard_normal((T, d)), r.standard_normal((T, dv)), r.standard_normal((T, d))
    want = np.stack([sum((q[t] @ k[s]) * a ** (t - s) * v[s] for s in range(t + 1)) for t in range(T)])
    assert np.allclose(plain.fixed_decay_scan(a, k, v, q), want)


def test_plain_router_groups():
    """A group counts by its two best together: one very good expert beside a bad one loses to two good ones, excluded experts
    do not come back although every choice score is negative, and a group of one counts by that one."""
    choice = np.array([-0.1, -0.9, -0.3, -0.35, -0.5, -0.45])
    assert plain.choose_experts(choice, 2, {"count": 3, "keep": 1}) == [2, 3]
    assert plain.choose_experts(choice, 3, {"count": 3, "keep": 2}) == [2, 3, 5]
    assert plain.choose_experts(choice, 2, None) == [0, 2]
    assert plain.choose_experts(choice, 2, {"count": 6, "keep": 3}) == [0, 2]
    assert plain.choose_experts(np.zeros(6), 2, {"count": 2, "keep": 1}) == [0, 1]


def test_plain_sink_takes_its_share():
    p = plain.softmax_with_sink(np.array([[0.0, 0.0, -np.inf]]), np.log(2.0))
    assert np.allclose(p, [[0.25, 0.25, 0.0]])
    assert np.allclose(plain.softmax_with_sink(np.array([[1.0, 2.0]]), 700.0), 0.0)


def test_the_mechanisms_matter(folders):
    """With these weights a limit, a sink, a pass's vector, a decay, the keep count or the rotation's scaling left out or
    changed moves the logits by far more than the tolerance."""
    c, W = plain.read_folder(folders["odd"])
    ids = requests(211, [40], seed=3)["r0"]
    base = plain.forward(c, W, ids)

    def differs(cfg, weights):
        return np.abs(plain.forward(cfg, weights, ids) - base).max() > 0.01 * np.abs(base).max()
    for edit in (lambda d: d["layers"][0]["mlp"]["expert"].update(limit=1e9), lambda d: d["layers"][1]["mlp"]["shared"].update(limit=1e9),
                 lambda d: d["layers"][0]["mixer"].update(decay=[0.9, 0.98, 0.999, 0.4, 0.99]), lambda d: d["loop"].update(times=1),
                 lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=3), lambda d: d["layers"][1]["mixer"]["rot"].pop("scaling"),
                 lambda d: d["layers"][3]["mixer"].update(scale=0.5)):
        d = copy.deepcopy(c)
        edit(d)
        assert differs(d, W)
    for name in ("l1.mix.sink", "l3.mix.sink", "loop.step", "l0.mlp.correction"):
        assert differs(c, dict(W, **{name: np.zeros_like(W[name]) - (50.0 if name.endswith("sink") else 0.0)})), name


@pytest.mark.parametrize("spec", [lightning(16, 20, (0.9997, 0.9999)), latent(4, 16, 8, 24, 32, 24, 1.5)])
def test_the_planted_token_decides(tmp_path, spec):
    """What the GPU tests of far tokens rest on: taking the planted token away moves the last position's logits a lot."""
    n, place = 90, 3
    folder = far_folder(spec, str(tmp_path), torch.float32, n, place, 149, 148)
    ids = [t % 147 for t in requests(150, [n], seed=6)["r0"]]
    ids[place], ids[-1] = 149, 148
    want = plain_logits(folder, ids)[-1]
    ids[place] = 147
    assert float((plain_logits(folder, ids)[-1] - want).abs().max()) > 0.25 * float(want.abs().max())
