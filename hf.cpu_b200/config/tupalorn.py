"""Tupalorn: a decoder of parallel layers (one norm, mixer and feed-forward read the same input) whose config.json lists its
layers one by one, with three kinds of mixer.

Top-level keys: ``architecture`` ("Tupalorn"), ``vocab``, ``width``, ``norm`` ({``eps``}), ``logit_softcap`` (logits pass through
``c tanh(z / c)``; absent: no cap) and ``layers``.  A layer entry has ``type`` (the kind of mixer), ``mixer`` (its sizes) and
``mlp`` (its feed-forward, or null for none):

* mixer "mamba2": ``heads``, ``vdim`` (value head), ``state`` (size of the state's other side), ``groups`` (of B and C; default
  1), ``conv`` (taps), ``norm_groups`` (equal parts of the output norm; default 1).  See ``parts/recurrent.py``.
* mixer "retention": ``heads``, ``dim`` (query/key head), ``vdim`` (value head; default: ``dim``), ``decay`` (a number per head),
  ``rot`` ({``dims``, ``base``}: rotation of the first ``dims`` dimensions of each query and key head, dimension i with i + dims/2;
  absent: none).
* mixer "attention": ``heads``, ``kv_heads`` (default: ``heads``), ``dim``, ``vdim`` (default: ``dim``), ``scale`` (factor on the
  scores), ``mask`` ({``size``}: a sliding window of that many positions, the query's own included; absent: causal), ``kv_from``
  (index of an earlier attention layer whose cached keys and values this layer reads; it then has none of its own).
  Queries and keys are normed over the whole projection; a gate of one number per head multiplies the heads' outputs.
* mlp ``kind`` "dense": ``ff``, ``limit``; with g and u the gate's and the up product's results (all products have biases),
  ``down(min(g, limit) sigmoid(1.702 min(g, limit)) (clamp(u, -limit, limit) + 1))``.

Every norm of the stream is a layer norm with a weight and no bias; the head is the embedding table.  Tensor names:
``embed``, ``l<i>.norm1``, ``l<i>.mix.{in,conv,conv.b,dt_bias,A_log,D,norm,o}``, or ``l<i>.mix.{q,k,v,g,o}``, or
``l<i>.mix.{q,k,v,g,o,q.norm,k.norm}``, ``l<i>.mlp.{gate,up,down}`` with ``.b``, ``final.norm``.

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
GATE_ALPHA, UP_OFFSET = 1.702, 1.0          # constants of the clamped gate that the design fixes


def _check_mixer(kind, m: Dict[str, Any], w: str) -> None:
    if kind == "mamba2":
        H, dv = take_int(m, "heads", lo=1), take_int(m, "vdim", lo=1)
        take_int(m, "state", lo=1), take_int(m, "conv", lo=1)
        G, parts = take_int(m, "groups", default=1, lo=1), take_int(m, "norm_groups", default=1, lo=1)
        if H % G:
            raise UnsupportedError(f"config.json: {w}{H} heads over {G} groups")
        if (H * dv) % parts:
            raise UnsupportedError(f"config.json: {w}{H * dv} channels in {parts} norm groups")
    elif kind == "retention":
        H, dim = take_int(m, "heads", lo=1), take_int(m, "dim", lo=1)
        take_int(m, "vdim", default=dim, lo=1)
        decay = m.get("decay")
        if not isinstance(decay, list) or len(decay) != H or any(isinstance(a, bool) or not isinstance(a, (int, float)) for a in decay):
            raise ConfigError(f"config.json: {w}'decay' must list one number for each of the {H} heads")
        if any(not 0 <= a <= 1 for a in decay):
            raise ConfigError(f"config.json: {w}'decay' must lie between 0 and 1")
        rot = _obj(m, "rot", w, required=False)
        if rot is not None:
            dims = take_int(rot, "dims", lo=0)
            if dims % 2 or dims > dim:
                raise UnsupportedError(f"config.json: {w}rot.dims {dims} must be even and at most {dim}")
            take_float(rot, "base", lo=0.0)
    elif kind == "attention":
        H = take_int(m, "heads", lo=1)
        G = take_int(m, "kv_heads", default=H, lo=1)
        if H % G:
            raise UnsupportedError(f"config.json: {w}unsupported attention geometry: {H} heads over {G} key/value heads")
        dim = take_int(m, "dim", lo=1)
        take_int(m, "vdim", default=dim, lo=1)
        take_float(m, "scale")
        mask = _obj(m, "mask", w, required=False)
        if mask is not None:
            take_int(mask, "size", lo=1)
    else:
        raise UnsupportedError(f"config.json: {w}mixer type '{kind}' is not supported (known: attention, mamba2, retention)")


def _heads(m):
    return m.get("kv_heads", m["heads"]), m["dim"], m.get("vdim", m["dim"])


def _window(m) -> int:
    return (m.get("mask") or {}).get("size", 0)


@dataclass
class TupalornConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm_eps: float = 1e-6
    logit_softcap: float = 0.0
    max_positions: int = DEFAULT_MAX_POSITIONS
    layers: List[Dict[str, Any]] = field(default_factory=list)
    eos_token_id: List[int] = field(default_factory=list)

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "TupalornConfig":
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
            m = _obj(L, "mixer", w)
            _check_mixer(L.get("type"), m, w)
            j = m.get("kv_from") if L["type"] == "attention" else None
            if j is not None:
                j = take_int(m, "kv_from", lo=0, hi=len(layers) - 1)
                if j >= i or layers[j].get("type") != "attention" or layers[j]["mixer"].get("kv_from") is not None:
                    raise ConfigError(f"config.json: {w}kv_from {j} is not an earlier attention layer with keys and values of its own")
                if _heads(layers[j]["mixer"]) != _heads(m):
                    raise ConfigError(f"config.json: {w}the key and value heads of layer {j} have other sizes")
            mlp = _obj(L, "mlp", w, required=False)
            if mlp is not None:
                if mlp.get("kind") != "dense":
                    raise UnsupportedError(f"config.json: {w}mlp kind '{mlp.get('kind')}' is not supported (known: dense)")
                take_int(mlp, "ff", lo=1)
                take_float(mlp, "limit", lo=0.0)
            out.append(copy.deepcopy(L))
        eos = d.get("eos_token_id", [])
        eos = [] if eos is None else ([eos] if isinstance(eos, int) else list(eos))
        return cls(vocab=V, width=E, norm_eps=take_float(norm, "eps", 1e-6, lo=0.0),
                   logit_softcap=take_float(d, "logit_softcap", default=0.0),
                   max_positions=take_int(d, "max_positions", default=DEFAULT_MAX_POSITIONS, lo=1), layers=out, eos_token_id=eos)

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture or "Tupalorn", "vocab": self.vocab, "width": self.width,
             "norm": {"eps": self.norm_eps}, "layers": copy.deepcopy(self.layers)}
        if self.logit_softcap:
            d["logit_softcap"] = self.logit_softcap
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_id:
            d["eos_token_id"] = list(self.eos_token_id)
        return d

    def cache_window(self, i: int) -> int:
        """The window layer i's cache keeps: the widest that it or a layer reading its keys and values sees (0: everything)."""
        sizes = [_window(self.layers[i]["mixer"])]
        sizes += [_window(L["mixer"]) for L in self.layers if L["type"] == "attention" and L["mixer"].get("kv_from") == i]
        return 0 if 0 in sizes else max(sizes)

    def plan(self) -> ModelPlan:
        E = self.width
        norm = lambda name: PartSpec("layernorm", {"size": E, "eps": self.norm_eps, "tensor": name})
        positions: Dict[str, PartSpec] = {}

        def rotary(rot, head_dim):
            # layers with the same rotation share one table
            if not rot or not rot["dims"]:
                return None
            name = f"rot{rot['dims']}_{float(rot['base'])!r}"
            positions.setdefault(name, PartSpec("rotary", {"head_dim": head_dim, "n_rot": rot["dims"], "theta": float(rot["base"]),
                                                           "pairing": "half"}))
            return name

        layers, schedule = [], []
        for i, L in enumerate(self.layers):
            p, m, mlp = f"l{i}", L["mixer"], L.get("mlp")
            common = {"hidden_size": E, "num_heads": m["heads"], "prefix": f"{p}.mix"}
            cache_of = None
            if L["type"] == "mamba2":
                mixer = PartSpec("mamba2", {**common, "v_head_dim": m["vdim"], "state_size": m["state"], "groups": m.get("groups", 1),
                                            "conv_taps": m["conv"], "norm_groups": m.get("norm_groups", 1), "norm_eps": self.norm_eps})
            elif L["type"] == "retention":
                mixer = PartSpec("retention", {**common, "head_dim": m["dim"], "v_head_dim": m.get("vdim", m["dim"]),
                                               "decay": [float(a) for a in m["decay"]], "norm_eps": self.norm_eps,
                                               "position": rotary(m.get("rot"), m["dim"])})
            else:
                cache_of = m.get("kv_from")
                window = _window(m)
                mixer = PartSpec("paged_attention", {
                    **common, "num_kv_heads": m.get("kv_heads", m["heads"]), "head_dim": m["dim"], "v_head_dim": m.get("vdim", m["dim"]),
                    "scale": float(m["scale"]), "qkv_bias": False, "out_bias": False, "window": window,
                    "cache_window": window if cache_of is not None else self.cache_window(i), "own_kv": cache_of is None,
                    "qk_norm_eps": self.norm_eps, "qk_row_norm": {"q": "q.norm", "k": "k.norm"}, "head_gate": "g", "position": None,
                    "names": {"q": "q", "k": "k", "v": "v", "o": "o"}, "weight_suffix": ""})
            ffn = None
            if mlp is not None:
                ffn = PartSpec("gated", {"hidden_size": E, "intermediate_size": mlp["ff"], "prefix": f"{p}.mlp", "activation": "clamped",
                                         "clamp": {"limit": float(mlp["limit"]), "alpha": GATE_ALPHA, "offset": UP_OFFSET},
                                         "bias_suffix": ".b", "names": {"gate": "gate", "up": "up", "down": "down"}})
            layers.append(LayerSpec(prefix=p, block=PartSpec("parallel_residual"), norm1=norm(f"{p}.norm1"), mixer=mixer, norm2=None, ffn=ffn))
            schedule.append(ScheduleEntry(i, cache_of))
        plan = ModelPlan(
            hidden_size=E, vocab_size=self.vocab, max_positions=self.max_positions,
            embedding=PartSpec("embedding", {"vocab_size": self.vocab, "hidden_size": E, "tensor": "embed"}),
            positions=positions, layers=layers, schedule=schedule, final_norm=norm("final.norm"),
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "hidden_size": E, "tensor": "embed", "softcap": self.logit_softcap}),
            eos_token_ids=list(self.eos_token_id))
        plan.validate()
        return plan


register_architecture("Tupalorn", TupalornConfig)
register_architecture("tupalorn", TupalornConfig)
