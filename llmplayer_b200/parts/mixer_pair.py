"""Two mixers side by side: both read the same input, and the layer's result is
left_scale * left(x) + right_scale * right(x) with two constants, each result optionally RMS-normed over the width first.

Each member is any registered mixer and keeps what it keeps (pages of keys and values, a recurrent state, ...); the pair
asks the cache for both (a :class:`BundleRequest`) and hands each member its own view. Where both members offer their
input projections (``offers_inputs``), one product forms both members' projections of the shared input. A member stores
its result in a float32 buffer (or adds it into a zeroed one, if it can only add); one kernel then norms both (if the
pair has norms), adds them, times their constants, into the stream and, with norms, writes the norm in front of the next
sublayer on the way. A member that leaves its output map's additive vector to the caller (``bias_later``) has it added
in that kernel too.
"""
from __future__ import annotations

import inspect
from typing import Dict, Mapping, Optional

import torch

from ..cache.sequence_cache import BundleRequest
from ..errors import ConfigError
from ..kernels import ops
from .base import MIXERS, NORMS, Part, PendingNorm, Runtime
from .linear import Linear
from .specs import MixerPairSpec, TensorSpec


class MixerPair(Part):
    def __init__(self, spec: MixerPairSpec):
        self.spec = spec
        self.left = MIXERS.build(spec.left)
        self.right = MIXERS.build(spec.right)
        if (spec.left_norm is None) != (spec.right_norm is None):
            raise ConfigError("both results of a pair are normed, or neither")
        self.norms = tuple(NORMS.build(n) for n in (spec.left_norm, spec.right_norm) if n is not None)
        for norm in self.norms:
            if not getattr(norm, "fusable_rms", False):
                raise ConfigError("the norms of a pair's results are RMS norms over whole rows")
        self.stacked = all(bool(getattr(m, "offers_inputs", False)) for m in (self.left, self.right))
        self.proj: Optional[Linear] = None
        self._right_at = 0
        call = "forward_projected" if self.stacked else "forward"
        self._args = [inspect.signature(getattr(m, call)).parameters for m in (self.left, self.right)]

    def children(self):
        return (self.left, self.right) + self.norms

    @property
    def capture_safe(self) -> bool:
        return all(bool(getattr(m, "capture_safe", False)) for m in self.children())

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        out: Dict[str, TensorSpec] = {}
        for m in self.children():
            out.update(m.tensor_specs())
        return out

    def load(self, tensors: Mapping[str, torch.Tensor], runtime: Runtime) -> None:
        super().load(tensors, runtime)
        for m in (self.left, self.right):
            if self.stacked:
                m.inputs_stacked = True
        for m in self.children():
            m.load(tensors, runtime)
        if self.stacked:
            left, right = self.left.take_inputs(), self.right.take_inputs()
            self._right_at = sum(int(w.shape[0]) for w in left)
            self.proj = Linear(left + right, runtime)

    def cache_request(self):
        return BundleRequest((self.left.cache_request(), self.right.cache_request()))

    def buffer_to_clear(self, ctx, tokens: int):
        if self.stacked:
            return self.proj.sums_into(ctx, tokens, "mixer_proj", ops.STORE)
        ask = getattr(self.left, "buffer_to_clear", None)
        return ask(ctx, tokens) if ask is not None else None

    def _run(self, member, args, ctx, view, source, width: int, name: str, prefix: str):
        """Run a member into a float32 buffer of its own; ``source``: the input, or (projections, first column). Returns
        (buffer, the vector it left to the caller or None)."""
        stacked = isinstance(source, tuple)
        y = ctx.buffer(name, ((source[0] if stacked else source).shape[0], width), torch.float32)
        kwargs = {}
        if "overwrite" in args:
            kwargs["overwrite"] = True
        else:
            y.zero_()
        later = "bias_later" in args and "overwrite" in args and getattr(member, "output_bias", None) is not None
        if later:
            kwargs["bias_later"] = True
        with ops.section_prefix(prefix):
            if stacked:
                member.forward_projected(ctx, view, source[0], source[1], y, **kwargs)
            else:
                member.forward(ctx, view, source, y, **kwargs)
        return y, (member.output_bias if later else None)

    def forward(self, ctx, cache, x, residual: torch.Tensor, then_norm=None, overwrite: bool = False) -> bool:
        """Adds the pair's result into ``residual`` (``overwrite``: the stream is set to zero first); returns whether
        ``then_norm`` was written on the way."""
        if isinstance(x, PendingNorm):
            x = x.tensor()
        T, width = x.shape[0], residual.shape[1]
        views = cache.members if cache is not None else (None, None)
        if self.stacked:
            proj = ctx.buffer("mixer_proj", (T, self.proj.out_features), torch.float32)
            with ops.section("mixer.proj"):
                self.proj.store(x, proj, ctx)
            sources = ((proj, 0), (proj, self._right_at))
        else:
            sources = (x, x)
        if overwrite:
            residual.zero_()
        s = self.spec
        a, a_vec = self._run(self.left, self._args[0], ctx, views[0], sources[0], width, "pair_left", "left.")
        b, b_vec = self._run(self.right, self._args[1], ctx, views[1], sources[1], width, "pair_right", "right.")
        with ops.section("mixer.sum"):
            if not self.norms:
                ops.scaled_sum(residual, a, s.left_scale, b, s.right_scale, a_vector=a_vec, b_vector=b_vec)
                return False
            for y, vec in ((a, a_vec), (b, b_vec)):
                if vec is not None:
                    ops.stream_add(y, None, vec)
            left, right = self.norms
            parts = getattr(then_norm.norm, "rms_parts", 0) if then_norm is not None else 0
            if not parts:
                ops.pair_norm_add(a, left.weight, s.left_scale, left.spec.eps, b, right.weight, s.right_scale, right.spec.eps, residual)
                return False
            ops.pair_norm_add(a, left.weight, s.left_scale, left.spec.eps, b, right.weight, s.right_scale, right.spec.eps, residual,
                              next_weight=then_norm.norm.weight, next_eps=then_norm.norm.spec.eps, next_parts=parts,
                              next_out=then_norm.out, clear=then_norm.clear)
            return True


MIXERS.register("mixer_pair", MixerPair)
