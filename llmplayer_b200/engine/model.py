"""A model: the parts of a layout, built, loaded and run in the schedule's order.

Reference: inference/InferenceEngine.java:53-101 builds the parts once;
:193-270 runs embedding, every layer, final norm and head for one token. Here
the same walk takes all tokens of a step at once, and the order of layers is the
layout's list of runs (a layer may run twice, or attend over an earlier run's cache).
"""
from __future__ import annotations

import inspect
from typing import Dict, List, Mapping, Optional

import torch

from ..errors import ConfigError
from ..parts import BLOCKS
from ..parts.base import Runtime
from ..parts.embedding import Embedding, LinearHead
from ..kernels import ops
from ..parts.specs import BIAS, ModelLayout, TensorSpec


class Model:
    def __init__(self, layout: ModelLayout):
        self.layout = layout
        self.embedding = Embedding(layout.embedding)
        self.blocks = [BLOCKS.build(spec) for spec in layout.layers]
        self.head = LinearHead(layout.head)
        self.runs = layout.run_order()
        for i, run in enumerate(self.runs):
            if not 0 <= run.layer < len(self.blocks):
                raise ConfigError(f"run {i} names layer {run.layer}, the model has {len(self.blocks)}")
            if run.reads_cache_of is not None and not 0 <= run.reads_cache_of < i:
                raise ConfigError(f"run {i} reads the cache of run {run.reads_cache_of}, which does not precede it")
            if i and (run.add_embedding or run.add_vector is not None) and all(
                    getattr(self.blocks[r.layer], "kind_bundle", False) for r in (self.runs[i - 1], run)):
                raise ConfigError(f"run {i} adds to the stream between two layers that keep a bundle of streams")
        self._check_shown_values()
        self.runtime: Optional[Runtime] = None
        # what some runs add to the stream before they start: the embedding's output, a row of a learned table
        self._keeps_embedding = any(run.add_embedding for run in self.runs)
        self._vector_rows: Dict[str, int] = {}
        for run in self.runs:
            if run.add_vector is not None:
                if run.add_row < 0:
                    raise ConfigError(f"row {run.add_row} of {run.add_vector!r}")
                self._vector_rows[run.add_vector] = max(self._vector_rows.get(run.add_vector, 0), run.add_row + 1)
        self._vectors: Dict[str, torch.Tensor] = {}
        # blocks whose forward takes (normed_ready, next_block) can hand a fused norm to the next block
        self._chains = ["next_block" in inspect.signature(b.forward).parameters for b in self.blocks]

    def _check_shown_values(self) -> None:
        """A layer that blends an earlier layer's values into its own finds them shown by a run before it, in its size."""
        shown = None
        for i, run in enumerate(self.runs):
            spec = getattr(self.layout.layers[run.layer], "mixer", None)
            size = getattr(spec, "num_kv_heads", 0) * (getattr(spec, "value_dim", None) or getattr(spec, "head_dim", 0))
            if getattr(spec, "value_blend", None) is not None and shown != size:
                raise ConfigError(f"run {i} blends {size} values per token, the runs before it show {shown or 'none'}")
            if getattr(spec, "shows_values", False):
                shown = size

    @property
    def capture_safe(self) -> bool:
        """Whether a captured graph of a one-token step may be replayed for other sequences: every part
        must read the step from device tensors only (``Part.capture_safe``)."""
        return all(bool(getattr(p, "capture_safe", False)) for p in [self.embedding, self.head] + self.blocks)

    # ------------------------------------------------------------------ tensors
    def tensor_specs(self) -> Dict[str, TensorSpec]:
        """Every tensor of the model folder, in a fixed order: embedding, layers, final norm, head."""
        out: Dict[str, TensorSpec] = {}
        parts = [self.embedding] + self.blocks + [self.head]
        for part in parts:
            for name, spec in part.tensor_specs().items():
                if name in out and out[name] != spec:
                    raise ConfigError(f"tensor {name!r} is asked for with shapes {out[name].shape} and {spec.shape}")
                out[name] = spec
        for name, rows in self._vector_rows.items():
            out[name] = TensorSpec((rows, self.layout.embedding.hidden_size), BIAS)
        return out

    def load(self, tensors: Mapping[str, torch.Tensor], runtime: Runtime) -> None:
        self.runtime = runtime
        self.embedding.load(tensors, runtime)
        for block in self.blocks:
            block.load(tensors, runtime)
        self.head.load(tensors, runtime)
        self._vectors = {name: runtime.gain(tensors[name]) for name in self._vector_rows}
        runtime.forget_uploads()

    # ------------------------------------------------------------------ cache
    def cache_requests(self) -> List[object]:
        """What each run keeps per sequence; a run that reads another's cache keeps nothing."""
        return [None if run.reads_cache_of is not None else self.blocks[run.layer].cache_request()
                for run in self.runs]

    def cache_owner(self, run_index: int) -> int:
        ref = self.runs[run_index].reads_cache_of
        return run_index if ref is None else ref

    # ------------------------------------------------------------------ a step
    def forward(self, ctx, cache, rows: torch.Tensor, logits: torch.Tensor) -> torch.Tensor:
        """Run the step's tokens through every run and fill ``logits[i]`` for token ``rows[i]``."""
        ctx.begin_walk()
        d = self.layout.embedding.hidden_size
        x = ctx.buffer("residual", (ctx.num_tokens, d), torch.float32)
        self.embedding.forward(ctx.tokens, x)
        x0 = None
        if self._keeps_embedding:
            x0 = ctx.buffer("embedding_out", (ctx.num_tokens, d), torch.float32)
            self.embedding.forward(ctx.tokens, x0)          # the rows again, into a buffer that the layers leave alone
        ready = False        # whether the previous block already normed the stream for this one
        for i, run in enumerate(self.runs):
            block = self.blocks[run.layer]
            if run.add_embedding or run.add_vector is not None:
                with ops.section("stream.add"):
                    ops.stream_add(x, x0 if run.add_embedding else None,
                                   self._vectors[run.add_vector][run.add_row] if run.add_vector is not None else None)
                ready = False
            following = self.blocks[self.runs[i + 1].layer] if i + 1 < len(self.runs) else None
            if following is not None and (self.runs[i + 1].add_embedding or self.runs[i + 1].add_vector is not None):
                following = None         # something is added to the stream before that run: its norm cannot be written yet
            if self._chains[run.layer]:
                ready = bool(block.forward(ctx, cache.view(self.cache_owner(i)), x, normed_ready=ready,
                                           next_block=following))
            else:
                block.forward(ctx, cache.view(self.cache_owner(i)), x)
                ready = False
        if rows.numel():
            self.head.forward(ctx, x, rows, logits)
        return logits


def expected_tensors(layout: ModelLayout) -> Dict[str, TensorSpec]:
    return Model(layout).tensor_specs()
