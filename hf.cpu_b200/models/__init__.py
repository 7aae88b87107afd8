"""A model put together from a plan: parts per layer, the run order, weights bound by name.

``Model.forward`` is the forward pass the step function drives: embedding, the schedule's
entries in order, then the final norm and the head on the rows whose logits are wanted
(src/model.c:545-640).
"""
from __future__ import annotations

import os
from dataclasses import dataclass
from typing import Dict, List, Optional

import torch

from ..config import ModelConfig, load_config
from ..config.base import ModelPlan
from ..parts import make_part
from ..weights import RandomSource, TensorSpec, load_tensors


EMBEDDING_STATE = "embedding"        # the key of the embedding's per-request state among the schedule entries' states


def block_state_key(entry: int):
    """The key of a block's own per-request state (a token shift's previous row) for schedule entry ``entry``; a layer
    that runs more than once has one per run."""
    return ("block", entry)


@dataclass
class Layer:
    block: object
    norm1: object
    mixer: object
    norm2: object
    ffn: object
    post1: object = None
    post2: object = None

    def parts(self):
        return tuple(p for p in (self.block, self.norm1, self.mixer, self.post1, self.norm2, self.ffn, self.post2)
                     if p is not None)

    def post_norms(self):
        """Keyword arguments for the block, for arrangements with norms behind the sublayers."""
        return {"post1": self.post1, "post2": self.post2} if self.post1 is not None else {}


class Model:
    def __init__(self, config: ModelConfig, run_dtype: torch.dtype = torch.bfloat16,
                 device: torch.device = torch.device("cuda:0"), plan: Optional[ModelPlan] = None):
        if run_dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"run dtype must be bfloat16 or float32, got {run_dtype}")
        self.config, self.run_dtype, self.device = config, run_dtype, torch.device(device)
        self.plan = plan if plan is not None else config.plan()
        self.plan.validate()
        p = self.plan
        self.positions = {name: make_part("position", spec) for name, spec in p.positions.items()}
        self.embedding = make_part("embedding", p.embedding)
        self.transitions = {name: make_part("transition", spec) for name, spec in p.transitions.items()}
        self.layers: List[Layer] = []
        for ls in p.layers:
            self.layers.append(Layer(
                block=make_part("block", ls.block),
                norm1=make_part("norm", ls.norm1),
                mixer=make_part("mixer", ls.mixer, positions=self.positions),
                norm2=make_part("norm", ls.norm2) if ls.norm2 is not None else None,
                ffn=make_part("ffn", ls.ffn) if ls.ffn is not None else None,
                post1=make_part("norm", ls.post_norm1) if ls.post_norm1 is not None else None,
                post2=make_part("norm", ls.post_norm2) if ls.post_norm2 is not None else None))
        self.final_norm = make_part("norm", p.final_norm)
        self.head = make_part("head", p.head)
        self.bound = False
        self.files: List[str] = []            # the weight files this model was loaded from

    # ---- weights ------------------------------------------------------------------------
    def all_parts(self):
        yield self.embedding
        yield from self.positions.values()
        yield from self.transitions.values()
        for l in self.layers:
            yield from l.parts()
        yield self.final_norm
        yield self.head

    def tensor_specs(self) -> List[TensorSpec]:
        seen: Dict[str, TensorSpec] = {}
        for part in self.all_parts():
            for s in part.tensor_specs():
                if s.name in seen and seen[s.name].shape != s.shape:
                    raise ValueError(f"tensor '{s.name}' is declared with two shapes")
                seen.setdefault(s.name, s)
        return list(seen.values())

    def bind(self, tensors) -> "Model":
        """Hand the weights to the parts.  ``tensors`` maps names to tensors: a dict, or a source that makes
        each tensor when it is asked for, so that the parts take them one at a time."""
        if hasattr(tensors, "keep"):
            # a tensor that two parts bind (a tied head reads the embedding) is made once
            count: Dict[str, int] = {}
            for part in self.all_parts():
                for s in part.tensor_specs():
                    count[s.name] = count.get(s.name, 0) + 1
            tensors.keep(n for n, c in count.items() if c > 1)
        for part in self.all_parts():
            part.bind(tensors, self.run_dtype, self.device)
        for l in self.layers:
            l.block.join_outputs(l.mixer, l.ffn)
        for pos in self.positions.values():
            pos.prepare(self.plan.max_positions, self.device)
        self.bound = True
        return self

    def weight_bytes_per_step(self) -> int:
        """Bytes of weights one decode step reads: every schedule entry's layer and the head, once each."""
        total = self.head.weight_bytes() + self.final_norm.weight_bytes()
        for e in self.plan.schedule:
            total += sum(p.weight_bytes() for p in self.layers[e.layer].parts())
            if e.enter is not None:
                total += self.transitions[e.enter[0]].weight_bytes()
        return total

    # ---- forward ------------------------------------------------------------------------
    def forward(self, ctx) -> Optional[torch.Tensor]:
        T = ctx.token_ids.shape[0]
        S = self.plan.streams
        x = ctx.buf("residual", (T, self.plan.hidden_size), torch.float32)
        self.embedding.forward(ctx.token_ids, x, ctx=ctx, state=ctx.entry_state(EMBEDDING_STATE))
        if S > 1:
            # the stream in S copies, a token's copies side by side, all equal to the embedding at the start
            emb, x = x, ctx.buf("residual_copies", (T, S * self.plan.hidden_size), torch.float32)
            from .. import kernels
            with kernels.phase("glue"):
                kernels.hc_spread(emb, x, S)
        schedule = self.plan.schedule
        for tr in self.transitions.values():
            tr.begin(ctx, x)
        xn = None                                # norm1 of the coming block, when the previous block computed it
        for i, e in enumerate(schedule):
            layer = self.layers[e.layer]
            owner = i if e.cache_of is None else e.cache_of
            # the norm that follows this block: the next block's first, or, after the last block of a step whose
            # tokens all want their logits (a step of single tokens), the final norm
            extra = layer.post_norms()
            if e.enter is not None:
                # (what the block in front handed over is the transition's operand; the layer's input comes out of it)
                out = ctx.buf("enter_xn", x.shape, self.run_dtype) if layer.block.state_spec() is None else None
                done = self.transitions[e.enter[0]].enter(ctx, x, e.enter[1], xn, layer.norm1 if out is not None else None, out)
                xn = out if done else None
            if i + 1 < len(schedule) and schedule[i + 1].enter is not None:
                next_norm = self.transitions[schedule[i + 1].enter[0]].operand_norm()
                if getattr(layer.block, "wants_next_block", False):
                    extra["next_block"] = None
            elif i + 1 < len(schedule):
                next_norm = self.layers[schedule[i + 1].layer].norm1
                following = self.layers[schedule[i + 1].layer].block
                if getattr(layer.block, "wants_next_block", False):
                    extra["next_block"] = following
                if following.state_spec() is not None:
                    # a block with state of its own (a token shift) makes its mixer's input itself, unless the block in
                    # front knows how to
                    if getattr(layer.block, "fuses_next_shift", False):
                        extra["next_block_state"] = ctx.entry_state(block_state_key(i + 1))
                    else:
                        next_norm = None
            else:
                next_norm = self.final_norm if getattr(ctx, "logits_for_all", False) else None
            if layer.block.state_spec() is not None:
                extra["block_state"] = ctx.entry_state(block_state_key(i))
            xn = layer.block.forward(ctx, x, layer.norm1, layer.mixer, layer.norm2, layer.ffn,
                                     ctx.entry_cache(owner), ctx.entry_state(i), e.cache_of is None,
                                     xn_ready=xn, next_norm=next_norm, **extra)
        M = ctx.num_logit_rows
        if M == 0:
            return None
        if xn is None or not schedule:
            xn = ctx.buf("head_xn", (M, self.plan.hidden_size), self.run_dtype)
            if S > 1:
                # the head reads the sum of the copies
                from .. import kernels
                params = getattr(self.final_norm, "params", None)
                with kernels.phase("glue"):
                    if params is not None:
                        kernels.hc_in_norm(x, S, None, ctx.logit_rows, params, xn)
                    else:
                        total = ctx.buf("head_sum", (M, self.plan.hidden_size), torch.float32)
                        kernels.hc_in_norm(x, S, None, ctx.logit_rows, None, total)
                        self.final_norm.forward(total, xn)
            else:
                self.final_norm.forward(x, xn, rows=ctx.logit_rows)
        logits = ctx.buf("logits", (M, self.plan.vocab_size), torch.float32)
        self.head.forward(xn, logits)
        return logits


def build_model_specs(config: ModelConfig) -> List[TensorSpec]:
    return Model(config, torch.float32, torch.device("cpu")).tensor_specs()


def load_model(path: str, dtype: torch.dtype = torch.bfloat16, device="cuda:0") -> Model:
    """Load a model folder (``config.json`` + safetensors: one file, or shards with or without an index) or one of
    the reference's GGUF files; the model class follows the configuration.  Every tensor is checked against the
    model's declaration before any is read, and tensors go to the device one at a time."""
    if os.path.isfile(path) and path.endswith(".gguf"):
        return load_gguf_model(path, dtype, device)
    config = load_config(path)
    model = Model(config, dtype, torch.device(device))
    tensors = load_tensors(path, model.tensor_specs(), dtype, model.device)
    try:
        model.bind(tensors)
        model.files = tensors.paths()
    finally:
        tensors.close()
    return model


def load_gguf_model(path: str, dtype: torch.dtype = torch.bfloat16, device="cuda:0") -> Model:
    """The same from one of the reference's own GGUF files (float tensor types only)."""
    from ..weights.gguf import GgufSource
    tensors = GgufSource(path, dtype, torch.device(device))
    try:
        model = Model(tensors.config, dtype, torch.device(device))
        tensors.check(model.tensor_specs())
        model.bind(tensors)
        model.files = [path]
    finally:
        tensors.close()
    return model


def random_model(config: ModelConfig, seed: int = 0, dtype: torch.dtype = torch.bfloat16, device="cuda:0",
                 std: float = 0.02) -> Model:
    """A model with random weights made directly on ``device`` (no files), one tensor at a time."""
    model = Model(config, dtype, torch.device(device))
    store = torch.float32 if dtype == torch.float32 else torch.bfloat16
    return model.bind(RandomSource(model.tensor_specs(), seed, store, model.device, std=std))
