"""Retention: linear attention with a fixed decay per head, without softmax or denominator.

    S_t = decay[h] S_(t-1) + k_t v_t^T;   o_t = S_t^T q_t          (S: [key_dim, value_dim], float32, zero at the start)

with queries and keys rotated by their position and keys times key_dim^-1/2. Each head's o_t is divided by its root mean
square (no gain), the heads are multiplied by silu(W_g x_t) and projected. The recurrence is one more form of the
framework's linear-attention scan (csrc/linear_attention.cu): one constant decay per head, queries and keys rotated as
the scan reads them from the projection (the cosines and sines of a step's tokens are formed once and shared by its
layers), long prompts in chunks side by side. The constant key_dim^-1/2 is applied to the queries, which gives the same
outputs; one-token steps run from the projection to the gated heads in one kernel (csrc/recurrent_step.cu). What a sequence carries from step to step is S. All kernels read the step from device tensors.
"""
from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from ..cache.sequence_cache import StateRequest
from ..errors import ConfigError
from ..kernels import ops
from .base import MIXERS, POSITIONS, Part, PendingNorm, Runtime
from .linear import Linear
from .specs import MATRIX, RetentionSpec, TensorSpec


class Retention(Part):
    def __init__(self, spec: RetentionSpec):
        s = spec
        if s.num_heads <= 0 or s.key_dim <= 0 or s.value_dim <= 0:
            raise ConfigError(f"retention with {s.num_heads} heads of {s.key_dim} x {s.value_dim}")
        if len(s.decays) != s.num_heads:
            raise ConfigError(f"{len(s.decays)} decays for {s.num_heads} heads")
        self.spec = spec
        self.position = POSITIONS.build(s.position)
        self.keys, self.values = s.num_heads * s.key_dim, s.num_heads * s.value_dim
        self.in_features = 2 * self.keys + 2 * self.values
        self.proj: Optional[Linear] = None
        self.out: Optional[Linear] = None
        self.inputs_stacked = False         # set by an owner whose one product covers this part's inputs
        self._inputs = []

    @property
    def capture_safe(self) -> bool:
        return bool(getattr(self.position, "capture_safe", False))

    # ------------------------------------------------------------------ tensors
    def tensor_specs(self) -> Dict[str, TensorSpec]:
        s = self.spec
        d = s.hidden_size
        return {
            s.q: TensorSpec((self.keys, d), MATRIX), s.k: TensorSpec((self.keys, d), MATRIX),
            s.v: TensorSpec((self.values, d), MATRIX), s.gate: TensorSpec((self.values, d), MATRIX),
            s.o: TensorSpec((d, self.values), MATRIX),
        }

    def load(self, tensors: Mapping[str, torch.Tensor], runtime: Runtime) -> None:
        super().load(tensors, runtime)
        s = self.spec
        self._inputs = [tensors[n] for n in (s.q, s.k, s.v, s.gate)]
        if not self.inputs_stacked:
            self.proj = Linear(self._inputs, runtime)
            self._inputs = []
        self.out = Linear([tensors[s.o]], runtime)
        self.decays = torch.tensor(s.decays, dtype=torch.float64).to(torch.float32).to(runtime.device)
        self.position.load(tensors, runtime)

    # ------------------------------------------------------------------ cache
    def cache_request(self):
        s = self.spec
        return StateRequest((s.num_heads, s.value_dim, s.key_dim), torch.float32)     # [head, value column, key channel]

    # ------------------------------------------------------------------ step
    offers_inputs = True

    def take_inputs(self):
        """The matrices that multiply the part's input, for an owner that set ``inputs_stacked`` before the load."""
        taken, self._inputs = self._inputs, []
        return taken

    def buffer_to_clear(self, ctx, tokens: int):
        return self.proj.sums_into(ctx, tokens, "mixer_proj", ops.STORE)

    def forward(self, ctx, cache, x, residual: torch.Tensor, then_norm=None, overwrite: bool = False) -> bool:
        """Adds the mixer's output into ``residual`` (``overwrite``: stores it there instead); returns whether
        ``then_norm`` was fused."""
        if isinstance(x, PendingNorm):
            x = x.tensor()
        proj = ctx.buffer("mixer_proj", (x.shape[0], self.proj.out_features), torch.float32)
        with ops.section("recurrence.proj"):
            self.proj.store(x, proj, ctx)
        return self.forward_projected(ctx, cache, proj, 0, residual, then_norm=then_norm, overwrite=overwrite)

    def forward_projected(self, ctx, cache, proj: torch.Tensor, offset: int, residual: torch.Tensor, then_norm=None,
                          overwrite: bool = True) -> bool:
        """From the input projections on: ``proj`` float32 [T, F] holds queries, keys, values and gate from column
        ``offset``."""
        s, rt = self.spec, self.runtime
        if cache is None:
            raise ConfigError("retention needs its per-sequence state")
        rotation = self.position.rotation()
        if rotation is None:
            raise ConfigError("retention applies rotations only (a position part with rotation())")
        T = proj.shape[0]
        H, dk, dv = s.num_heads, s.key_dim, s.value_dim
        v_off = offset + 2 * self.keys
        g_off = v_off + self.values
        o = ctx.buffer("attn_out", (T, self.values), rt.act_dtype)
        # an output product that sums partial results wants its target zero: the kernel before it clears it on the side
        clear = residual if overwrite and residual.dtype == torch.float32 and self.out.needs_zero(T) else None
        if ctx.all_single and dk + dv <= 5800:
            with ops.section("recurrence.step"):
                ops.retention_step(proj, (offset, offset + self.keys, v_off, g_off), rotation, ctx.positions, self.decays, cache.rows,
                                   ctx.slots, s.norm_eps, o, num_heads=H, key_dim=dk, value_dim=dv, q_scale=float(dk) ** -0.5, clear=clear)
        else:
            raw = ctx.buffer("recurrence_raw", (T, self.values), torch.float32)
            self._scan(ctx, cache, proj, (offset, offset + self.keys, v_off), rotation, raw)
            with ops.section("recurrence.norm"):
                ops.gla_finish(raw, None, s.norm_eps, proj[:, g_off:g_off + self.values], o, num_heads=H, value_dim=dv, clear=clear)
        if clear is not None:
            ctx.note_cleared()
        with ops.section("recurrence.out"):
            if overwrite:
                self.out.store(o, residual, ctx)
                return False
            return self.out.accumulate(o, residual, ctx, then_norm)

    def _scan(self, ctx, cache, proj: torch.Tensor, columns, rotation, raw: torch.Tensor) -> None:
        s, rt = self.spec, self.runtime
        H, dk, dv = s.num_heads, s.key_dim, s.value_dim
        with ops.section("recurrence.scan"):
            ops.gla_scan(proj, *columns, self.decays, cache.rows, ctx.slots, ctx.q_start, raw,
                         num_heads=H, key_dim=dk, value_dim=dv, q_scale=float(dk) ** -0.5, max_new=ctx.max_new,
                         scratch=ctx.buffer, decay_fixed=True, rotation=rotation,
                         angles=ctx.angles(rotation) if rotation.rotary_dim else None, tensor_cores=rt.fast)


MIXERS.register("retention", Retention)
