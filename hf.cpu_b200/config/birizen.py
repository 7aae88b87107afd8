"""Birizen: a decoder with a norm on both sides of every sublayer, a routed feed-forward in its layers, two kinds of mixer, and
a stretch of layers that runs several times and reads the embedding again in front of every pass.

Top-level keys: ``architecture`` ("Birizen"), ``vocab``, ``width``, ``norm`` ({``eps``}), ``layers`` and optionally ``loop``
({``start``, ``stop``, ``times``}: layers start .. stop - 1 run ``times`` times in a row with the same weights, each pass with
caches and states of its own, and in front of each pass the stream becomes ``W_in [x; x0] + step_t``, x0 being the embedding
output; then the rest follow).  A layer entry has ``type`` (the kind of mixer), ``mixer`` (its sizes) and ``mlp`` (its
feed-forward, or null for none):

* mixer "lightning": ``heads``, ``dim`` (query/key head), ``vdim`` (value head; default: ``dim``), ``decay`` (a number per
  head).  Linear attention with a fixed decay per head on silu(q), silu(k), silu(v); the heads are normed together and gated
  with a sigmoid (see ``parts/recurrent.py``).
* mixer "latent_attention": ``heads``, ``dim`` (plain) and ``rot_dim`` (rotated) dimensions per query/key head, ``vdim``
  (default: ``dim``), ``q_rank`` and ``kv_rank`` (the latents), ``scale``, ``rot`` ({``dims`` = ``rot_dim``, ``base``, optionally
  ``scaling``: {``factor``, ``original``, ``fast``, ``slow``}}: pairs (2i, 2i + 1)); causal, a learned sink per head, an
  element-wise sigmoid gate on the heads.
* mlp ``kind`` "moe": ``expert`` ({``ff``, ``limit``}), ``router`` ({``experts``, ``top``, optionally ``groups``: {``count``,
  ``keep``}}) and optionally ``shared`` ({``ff``, ``limit``}).  Experts are ``down(g sigmoid(1.702 g) (u + 1))`` with g =
  min(gate x, limit), u = clamp(up x, -limit, limit); the router scores with a sigmoid and chooses with a stored correction.

Every norm is an RMSNorm with a plain weight; the head is the embedding table.  Tensor names: ``embed``, ``loop.in``,
``loop.step``, ``l<i>.norm1`` / ``norm1b`` / ``norm2`` / ``norm2b``, ``l<i>.mix.{q,k,v,g,o,norm}`` or ``l<i>.mix.{dq,uq,dkv,uk,uv,g,
o,sink}`` with ``dq.norm`` / ``dkv.norm``, ``l<i>.mlp.{router,correction}``, ``l<i>.mlp.{e<j>,shared}.{gate,up,down}``, ``final.norm``.

config.json gives no context length: ``max_positions`` (optional key, default below) bounds the rotary tables and a
request's length in this engine.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List

from .base import (ConfigError, LayerSpec, ModelConfig, ModelPlan, PartSpec, ScheduleEntry, UnsupportedError,
                   take_float, take_int)
from .manapel import _obj
from .registry import register_architecture

DEFAULT_MAX_POSITIONS = 1 << 16
SCALING_KEYS = ("factor", "original", "fast", "slow")
GATE_ALPHA, UP_OFFSET = 1.702, 1.0      # of the clamped gated feed-forward


def _check_lightning(m: Dict[str, Any], w: str) -> None:
    H = take_int(m, "heads", lo=1)
    d = take_int(m, "dim", lo=1)
    take_int(m, "vdim", default=d, lo=1)
    decay = m.get("decay")
    if not isinstance(decay, list) or len(decay) != H or not all(
            isinstance(a, (int, float)) and not isinstance(a, bool) and 0.0 <= a <= 1.0 for a in decay):
        raise ConfigError(f"config.json: {w}decay must be {H} numbers between 0 and 1, one per head")


def _check_latent(m: Dict[str, Any], w: str) -> None:
    take_int(m, "heads", lo=1)
    d = take_int(m, "dim", lo=1)
    take_int(m, "vdim", default=d, lo=1)
    take_int(m, "q_rank", lo=1), take_int(m, "kv_rank", lo=1)
    take_float(m, "scale")
    rd = take_int(m, "rot_dim", lo=0)
    if rd % 2:
        raise UnsupportedError(f"config.json: {w}rot_dim {rd} must be even")
    if rd:
        rot = _obj(m, "rot", w)
        if take_int(rot, "dims", lo=2) != rd:
            raise UnsupportedError(f"config.json: {w}rot.dims must equal rot_dim (the rotated part is rotated whole)")
        take_float(rot, "base", lo=0.0)
        sc = _obj(rot, "scaling", w, required=False)
        if sc is not None:
            for k in SCALING_KEYS:
                take_float(sc, k, lo=0.0)


def _check_mlp(mlp: Dict[str, Any], w: str) -> None:
    if mlp.get("kind") != "moe":
        raise UnsupportedError(f"config.json: {w}mlp kind '{mlp.get('kind')}' is not supported (known: moe)")
    e = _obj(mlp, "expert", w)
    take_int(e, "ff", lo=1), take_float(e, "limit", lo=0.0)
    r = _obj(mlp, "router", w)
    n, top = take_int(r, "experts", lo=1), take_int(r, "top", lo=1)
    if top > n:
        raise ConfigError(f"config.json: {w}router.top {top} exceeds the {n} experts")
    g = _obj(r, "groups", w, required=False)
    if g is not None:
        count, keep = take_int(g, "count", lo=1), take_int(g, "keep", lo=1)
        if n % count or keep > count or keep * (n // count) < top:
            raise ConfigError(f"config.json: {w}router.groups: {count} groups of which {keep} are kept do not fit {n} experts "
                              f"with top {top}")
    shared = _obj(mlp, "shared", w, required=False)
    if shared is not None:
        take_int(shared, "ff", lo=1), take_float(shared, "limit", lo=0.0)


@dataclass
class BirizenConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm_eps: float = 1e-6
    max_positions: int = DEFAULT_MAX_POSITIONS
    layers: List[Dict[str, Any]] = field(default_factory=list)
    loop: Dict[str, int] = field(default_factory=dict)          # start, stop, times; empty: every layer runs once
    eos_token_id: List[int] = field(default_factory=list)

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "BirizenConfig":
        V = take_int(d, "vocab", lo=1)
        E = take_int(d, "width", lo=1, hi=1_000_000)
        norm = _obj(d, "norm", "")
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        out = []
        for i, L in enumerate(layers):
            w = f"layers[{i}]: "
            if not isinstance(L, dict):
                raise ConfigError(f"config.json: {w}must be an object")
            kind, m = L.get("type"), _obj(L, "mixer", w)
            if kind == "lightning":
                _check_lightning(m, w)
            elif kind == "latent_attention":
                _check_latent(m, w)
            else:
                raise UnsupportedError(f"config.json: {w}mixer type '{kind}' is not supported (known: latent_attention, lightning)")
            mlp = _obj(L, "mlp", w, required=False)
            if mlp is not None:
                _check_mlp(mlp, w)
            out.append(copy.deepcopy(L))
        loop = _obj(d, "loop", "", required=False)
        lp: Dict[str, int] = {}
        if loop is not None:
            lp = {"start": take_int(loop, "start", lo=0), "stop": take_int(loop, "stop", lo=0), "times": take_int(loop, "times", lo=0)}
            if not lp["start"] <= lp["stop"] <= len(out):
                raise ConfigError(f"config.json: loop: layers {lp['start']} .. {lp['stop']} are not a stretch of the {len(out)} layers")
        eos = d.get("eos_token_id", [])
        eos = [] if eos is None else ([eos] if isinstance(eos, int) else list(eos))
        return cls(vocab=V, width=E, norm_eps=take_float(norm, "eps", 1e-6, lo=0.0),
                   max_positions=take_int(d, "max_positions", default=DEFAULT_MAX_POSITIONS, lo=1), layers=out, loop=lp,
                   eos_token_id=eos)

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture or "Birizen", "vocab": self.vocab, "width": self.width,
             "norm": {"eps": self.norm_eps}, "layers": copy.deepcopy(self.layers)}
        if self.loop:
            d["loop"] = dict(self.loop)
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_id:
            d["eos_token_id"] = list(self.eos_token_id)
        return d

    def run_order(self) -> List[ScheduleEntry]:
        """The layers in the order they run; the first layer of a pass enters through the loop's transition."""
        n = len(self.layers)
        if not self.loop:
            return [ScheduleEntry(i) for i in range(n)]
        a, b, times = self.loop["start"], self.loop["stop"], self.loop["times"]
        passes = [ScheduleEntry(i, enter=("loop", t) if i == a else None) for t in range(times) for i in range(a, b)]
        return [ScheduleEntry(i) for i in range(a)] + passes + [ScheduleEntry(i) for i in range(b, n)]

    def _mixer(self, L, p, positions) -> PartSpec:
        m = L["mixer"]
        if L["type"] == "lightning":
            return PartSpec("lightning_attention", {
                "hidden_size": self.width, "num_heads": m["heads"], "head_dim": m["dim"], "v_head_dim": m.get("vdim", m["dim"]),
                "decay": [float(a) for a in m["decay"]], "norm_eps": self.norm_eps, "prefix": f"{p}.mix", "activation": "silu",
                "key_scale": 1.0, "norm_tensor": "norm", "gate": "sigmoid"})
        pos_name = None
        if m["rot_dim"]:
            rot = m["rot"]
            sc = rot.get("scaling")
            # layers with the same rotation share one table
            pos_name = f"rot{rot['dims']}_{float(rot['base'])!r}_{sorted(sc.items()) if sc else None!r}"
            positions.setdefault(pos_name, PartSpec("rotary", {
                "head_dim": m["rot_dim"], "n_rot": rot["dims"], "theta": float(rot["base"]), "pairing": "interleaved",
                "scaling": {k: float(sc[k]) for k in SCALING_KEYS} if sc else None}))
        return PartSpec("latent_attention", {
            "hidden_size": self.width, "num_heads": m["heads"], "head_dim": m["dim"], "rot_dim": m["rot_dim"],
            "v_head_dim": m.get("vdim", m["dim"]), "q_rank": m["q_rank"], "kv_rank": m["kv_rank"], "scale": float(m["scale"]),
            "norm_eps": self.norm_eps, "window": 0, "position": pos_name, "prefix": f"{p}.mix", "sink_tensor": "sink",
            "gate_tensor": "g"})

    def _ffn(self, mlp, p) -> PartSpec:
        e, r, shared = mlp["expert"], mlp["router"], mlp.get("shared")
        g = r.get("groups")
        clamp = lambda limit: {"limit": float(limit), "alpha": GATE_ALPHA, "offset": UP_OFFSET}
        return PartSpec("moe", {
            "hidden_size": self.width, "experts": r["experts"], "top": r["top"], "expert_size": e["ff"], "prefix": f"{p}.mlp",
            "activation": "clamped", "clamp": clamp(e["limit"]), "gated": True, "router_bias": False, "router": "sigmoid",
            "correction": "correction", "groups": (g["count"], g["keep"]) if g else None, "group_best": 2, "renorm": True,
            "shared_size": shared["ff"] if shared else 0, "shared_clamp": clamp(shared["limit"]) if shared else None,
            "names": {"router": "router", "expert": "e{}", "shared": "shared", "gate": "gate", "up": "up", "down": "down"}})

    def plan(self) -> ModelPlan:
        E = self.width
        norm = lambda name, optional=False: PartSpec("rmsnorm", {"size": E, "eps": self.norm_eps, "tensor": name, "optional": optional})
        positions: Dict[str, PartSpec] = {}
        layers = []
        for i, L in enumerate(self.layers):
            p, mlp = f"l{i}", L.get("mlp")
            none = mlp is None
            layers.append(LayerSpec(
                prefix=p, block=PartSpec("sandwich_residual"), norm1=norm(f"{p}.norm1"), mixer=self._mixer(L, p, positions),
                norm2=norm(f"{p}.norm2", none), ffn=None if none else self._ffn(mlp, p),
                post_norm1=norm(f"{p}.norm1b"), post_norm2=norm(f"{p}.norm2b", none)))
        transitions = {}
        if self.loop:
            transitions["loop"] = PartSpec("join_embedding", {
                "hidden_size": E, "passes": self.loop["times"], "tensor": "loop.in", "step_tensor": "loop.step",
                "first": self.loop["start"] == 0})
        plan = ModelPlan(
            hidden_size=E, vocab_size=self.vocab, max_positions=self.max_positions,
            embedding=PartSpec("embedding", {"vocab_size": self.vocab, "hidden_size": E, "tensor": "embed"}),
            positions=positions, layers=layers, schedule=self.run_order(), final_norm=norm("final.norm"),
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "hidden_size": E, "tensor": "embed"}),
            eos_token_ids=list(self.eos_token_id), transitions=transitions)
        plan.validate()
        return plan


register_architecture("Birizen", BirizenConfig)
register_architecture("birizen", BirizenConfig)
