"""A matrix state per head updated by the gated delta rule.

Queries and keys (``num_qk_heads`` heads of ``key_dim``) and values (``num_heads`` heads of ``value_dim``) each pass a
short causal convolution per channel and silu; queries and keys are then made unit vectors per head (queries also times
key_dim^-1/2). Per head h, which reads query / key head h // (num_heads // num_qk_heads):

    b_t = sigmoid(W_b x_t)                                  g_t = exp(-exp(a_log[h]) * softplus(W_a x_t + dt_bias[h]))
    S <- g_t S;   u = b_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t          (S: [key_dim, value_dim])

so the read-out sees the token's own write. The decay may also differ from key channel to key channel: g_t is then the
diagonal of exp(-exp(a_log[h]) * softplus(U (D x_t) + dt_bias)) with a low-rank map U D of the input, and the output gate
may be the sigmoid of another low-rank map instead of silu(W_g x_t). Each head's o_t is divided by its root mean square, multiplied by a gain
shared by the heads and by silu(W_g x_t), and projected. State, decays, strengths, unit norms and every sum are float32.
The recurrence is one more form of the framework's linear-attention scan (csrc/linear_attention.cu): a value column's
state entries live in the registers of a few threads, and the two read-outs S^T k and S^T q of a token are taken from
the state before it in one pass of shuffles. Prompts of bfloat16 models run in chunks of 32 tokens whose sums are
tensor-core products at float32 precision (csrc/chunked_recurrence.cu); steps of one token per sequence run from the
projection to the gated heads in one kernel (csrc/recurrent_step.cu). float32 prompts of 256 tokens or more run in chunks
side by side (a chunk's effect on the state that enters it is S -> P S + L; the first pass forms P, a [key_dim, key_dim]
matrix, beside L, the chunks' start states follow in order, the second pass writes the outputs). What a sequence carries
from step to step is S and the convolutions' last taps - 1 inputs. All kernels read the step from device tensors.
"""
from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from ..cache.sequence_cache import StateRequest
from ..errors import ConfigError, WeightError
from ..kernels import ops
from .base import MIXERS, Part, PendingNorm, Runtime
from .linear import Linear
from .specs import ANY, BIAS, GAIN, MATRIX, GatedDeltaRuleSpec, TensorSpec

UNIT_EPS = 1e-6         # inside the root of the heads' unit norm: the design fixes it


class GatedDeltaRule(Part):
    capture_safe = True

    def __init__(self, spec: GatedDeltaRuleSpec):
        s = spec
        if s.num_heads <= 0 or s.num_qk_heads <= 0 or s.num_heads % s.num_qk_heads:
            raise ConfigError(f"{s.num_heads} heads cannot share {s.num_qk_heads} query / key heads")
        if s.key_dim <= 0 or s.value_dim <= 0:
            raise ConfigError(f"a delta rule with heads of {s.key_dim} x {s.value_dim}")
        if not 1 <= s.conv_taps <= 8:
            raise ConfigError(f"a convolution of {s.conv_taps} taps (supported: 1 to 8)")
        if s.gate_activation not in ("silu", "sigmoid"):
            raise ConfigError(f"unknown activation {s.gate_activation!r} of a delta rule's output gate")
        if s.gate_up is not None and s.decay_up is None:
            raise ConfigError("a low-rank output gate comes with low-rank decays")
        self.spec = spec
        self.qk = s.num_qk_heads * s.key_dim
        self.values = s.num_heads * s.value_dim
        self.conv_channels = 2 * self.qk + self.values
        self.proj: Optional[Linear] = None
        self.out: Optional[Linear] = None
        self.inputs_stacked = False         # set by an owner whose one product covers this part's inputs
        self._inputs = []

    # ------------------------------------------------------------------ tensors
    def tensor_specs(self) -> Dict[str, TensorSpec]:
        s = self.spec
        d, H, K = s.hidden_size, s.num_heads, s.conv_taps
        return {
            s.q: TensorSpec((self.qk, d), MATRIX), s.q_conv: TensorSpec((self.qk, K), MATRIX),
            s.k: TensorSpec((self.qk, d), MATRIX), s.k_conv: TensorSpec((self.qk, K), MATRIX),
            s.v: TensorSpec((self.values, d), MATRIX), s.v_conv: TensorSpec((self.values, K), MATRIX),
            s.strength: TensorSpec((H, d), MATRIX),
            s.a_log: TensorSpec((H,), BIAS),
            s.out_norm: TensorSpec((s.value_dim,), GAIN),
            s.decay: TensorSpec((H if s.decay_up is None else ANY, d), MATRIX, fill=s.key_dim),
            s.dt_bias: TensorSpec((H if s.decay_up is None else H * s.key_dim,), BIAS),
            s.gate: TensorSpec((self.values if s.gate_up is None else ANY, d), MATRIX, fill=s.key_dim),
            s.o: TensorSpec((d, self.values), MATRIX),
            **({s.decay_up: TensorSpec((H * s.key_dim, ANY), MATRIX, fill=s.key_dim)} if s.decay_up is not None else {}),
            **({s.gate_up: TensorSpec((self.values, ANY), MATRIX, fill=s.key_dim)} if s.gate_up is not None else {}),
        }

    def load(self, tensors: Mapping[str, torch.Tensor], runtime: Runtime) -> None:
        super().load(tensors, runtime)
        s = self.spec
        # one product of the normed input: queries, keys, values (the convolution's channels, in this order), then the
        # write strength's and the decay's pre-activations and the output gate (or the low-rank factors of these two)
        self._inputs = [tensors[n] for n in (s.q, s.k, s.v, s.strength, s.decay, s.gate)]
        self.decay_rows, self.gate_rows = int(tensors[s.decay].shape[0]), int(tensors[s.gate].shape[0])
        self.in_features = sum(int(m.shape[0]) for m in self._inputs)
        if not self.inputs_stacked:
            self.proj = Linear(self._inputs, runtime)
            self._inputs = []
        for down, up in ((s.decay, s.decay_up), (s.gate, s.gate_up)):
            if up is not None and tensors[down].shape[0] != tensors[up].shape[1]:
                raise WeightError(f"{down} has {tensors[down].shape[0]} rows but {up} has {tensors[up].shape[1]} columns")
        self.decay_up = runtime.matrix(tensors[s.decay_up]) if s.decay_up is not None else None
        self.gate_up = runtime.matrix(tensors[s.gate_up]) if s.gate_up is not None else None
        if self.decay_up is not None and self.gate_up is not None and self.decay_up.dtype != self.gate_up.dtype:
            self.decay_up, self.gate_up = self.decay_up.float(), self.gate_up.float()       # mixed storage: widen
        # one token per sequence in one kernel, a CTA per query / key head; with many value heads on one it would be slow
        self.step_kernel = s.num_heads // s.num_qk_heads <= 4 and s.value_dim * 3 + s.key_dim * 3 + self.decay_rows + self.gate_rows <= 11000
        self.taps = runtime.gain(torch.cat([tensors[n].to(torch.float32) for n in (s.q_conv, s.k_conv, s.v_conv)], dim=0))
        self.a_log = runtime.gain(tensors[s.a_log])
        self.dt_bias = runtime.gain(tensors[s.dt_bias])
        self.out_gain = runtime.gain(tensors[s.out_norm])
        self.out = Linear([tensors[s.o]], runtime)

    # ------------------------------------------------------------------ cache
    def cache_request(self):
        s = self.spec
        return (StateRequest((s.num_heads, s.value_dim, s.key_dim), torch.float32),      # [head, value column, key channel]
                StateRequest((s.conv_taps - 1, self.conv_channels), torch.float32))

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
        """From the input projections on: ``proj`` float32 [T, F] holds them from column ``offset``, in the order of
        :meth:`take_inputs`."""
        s, rt = self.spec, self.runtime
        if cache is None:
            raise ConfigError("a delta rule needs its per-sequence state")
        T = proj.shape[0]
        H, G, dk, dv = s.num_heads, s.num_qk_heads, s.key_dim, s.value_dim
        C = self.conv_channels
        b_off = offset + C
        a_off = b_off + H
        g_off = a_off + self.decay_rows
        state, tail = cache.blocks
        o = ctx.buffer("attn_out", (T, self.values), rt.act_dtype)
        clear = residual if overwrite and residual.dtype == torch.float32 and self.out.needs_zero(T) else None
        if ctx.all_single and self.step_kernel:
            with ops.section("recurrence.step"):
                ops.delta_step(proj, (offset, b_off, a_off, g_off), self.taps, tail, state, ctx.slots, self.dt_bias, self.a_log,
                               self.out_gain, s.norm_eps, o, num_heads=H, qk_heads=G, key_dim=dk, value_dim=dv, unit_eps=UNIT_EPS,
                               q_scale=float(dk) ** -0.5, a_up=self.decay_up, g_up=self.gate_up,
                               gate_sigmoid=s.gate_activation == "sigmoid", clear=clear)
        else:
            self._recur(ctx, proj, offset, state, tail, o, clear)
        if clear is not None:
            ctx.note_cleared()
        with ops.section("recurrence.out"):
            if overwrite:
                self.out.store(o, residual, ctx)
                return False
            return self.out.accumulate(o, residual, ctx, then_norm)

    def _recur(self, ctx, proj: torch.Tensor, offset: int, state: torch.Tensor, tail: torch.Tensor, o: torch.Tensor, clear) -> None:
        """From the input projections to the normed and gated heads ``o``, for steps with several tokens of a sequence."""
        s, rt = self.spec, self.runtime
        T = proj.shape[0]
        H, G, dk, dv = s.num_heads, s.num_qk_heads, s.key_dim, s.value_dim
        C = self.conv_channels
        b_off = offset + C
        a_off = b_off + H
        g_off = a_off + self.decay_rows
        mixed = ctx.buffer("conv_out", (T, C), torch.float32)            # [q | k | v] behind the convolutions
        with ops.section("recurrence.conv"):
            ops.conv_unit_heads(proj[:, offset:offset + C], self.taps, tail, ctx.slots, ctx.q_start, mixed, max_new=ctx.max_new,
                                heads=2 * G, dim=dk, eps=UNIT_EPS, scale=float(dk) ** -0.5, scaled_heads=G)
        by_channel = self.decay_up is not None
        gate = proj[:, g_off:g_off + self.gate_rows]
        with ops.section("recurrence.gates"):
            strength = ctx.buffer("write_strengths", (T, H), torch.float32)
            if by_channel:
                decay = ctx.buffer("channel_decays", (T, H * dk), torch.float32)
                if self.gate_up is not None:
                    gate = ctx.buffer("output_gate", (T, self.values), torch.float32)
                ops.low_rank_gates(proj, a_off, self.decay_up, self.dt_bias, self.a_log, decay, b_off, strength, key_dim=dk,
                                   g_off=g_off, g_up=self.gate_up, gate=gate if self.gate_up is not None else None)
            else:
                decay = ctx.buffer("decay_gates", (T, H), torch.float32)
                ops.decay_gates(proj, a_off, self.dt_bias, self.a_log, decay, strength=strength, b_off=b_off)
        raw = ctx.buffer("recurrence_raw", (T, self.values), torch.float32)
        with ops.section("recurrence.scan"):
            ops.gla_scan(mixed, 0, self.qk, 2 * self.qk, decay, state, ctx.slots, ctx.q_start, raw, num_heads=H,
                         key_dim=dk, value_dim=dv, q_scale=1.0, max_new=ctx.max_new, scratch=ctx.buffer,
                         decay_per_head=not by_channel, qk_heads=G, delta_strength=strength, tensor_cores=rt.fast)
        with ops.section("recurrence.norm"):
            ops.gla_finish(raw, self.out_gain, s.norm_eps, gate, o, num_heads=H, value_dim=dv, clear=clear,
                           gate_sigmoid=s.gate_activation == "sigmoid")


MIXERS.register("gated_delta_rule", GatedDeltaRule)
