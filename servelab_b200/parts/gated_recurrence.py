"""A recurrent block with one number of state a channel (spec: ``GatedRecurrenceSpec``).

Per step, with h the mixer's input [T, hidden]:

  1. one product for both branches y | x (concatenated at load);
  2. the causal convolution of the x branch, its biases inside; a request's last ``conv_taps`` - 1 rows
     are part of its record;
  3. the gates' logits by block-diagonal products (both gates of a block in one matrix), float32;
  4. one kernel: gates, decays, the recurrence over the tokens of every request in order (float32, the
     state in the request's slot), times gelu_tanh of the y branch;
  5. the output projection.
"""

from __future__ import annotations

import torch

from ..cache.manager import FixedStateRequest
from ..ops import kernels as K
from ..ops.linear import block_diagonal_logits, linear
from ..weights.source import BIAS, MATRIX, TensorDecl
from .base import Mixer
from .normed_attention import pad_rows
from .registry import register_mixer


@register_mixer("gated_recurrence")
class GatedRecurrence(Mixer):
    graph_safe = True
    padded_steps_safe = True      # requests without tokens and tokens of no request leave the records alone

    def __init__(self, spec, prefix, env):
        super().__init__(spec, prefix, env)
        s = spec
        if min(s.width, s.blocks) <= 0 or s.width % s.blocks:
            raise ValueError("gated_recurrence: width must be a positive multiple of blocks")
        if not 1 <= s.conv_taps <= K.CONV_MAX_TAPS:
            raise ValueError(f"gated_recurrence: 1..{K.CONV_MAX_TAPS} taps, got {s.conv_taps}")
        if s.decay_coef < 0:
            raise ValueError("gated_recurrence: decay_coef must not be negative")
        self.out_dtype = None                  # (set by a mixer that wraps this one)
        self.state_floats = self._state_floats(s)

    @classmethod
    def _names(cls, spec, prefix):
        return {n: f"{prefix}.{getattr(spec, n + '_name')}" for n in ("y", "x", "conv", "r", "i", "lambda", "o")}

    @classmethod
    def declare(cls, spec, prefix):
        h, w, b = spec.hidden_size, spec.width, spec.blocks
        n, sfx = cls._names(spec, prefix), spec.bias_suffix
        out = [TensorDecl(n["y"], (w, h), MATRIX), TensorDecl(n["y"] + sfx, (w,), BIAS),
               TensorDecl(n["x"], (w, h), MATRIX), TensorDecl(n["x"] + sfx, (w,), BIAS),
               TensorDecl(n["conv"], (w, spec.conv_taps), BIAS), TensorDecl(n["conv"] + sfx, (w,), BIAS)]
        for g in ("r", "i"):
            out += [TensorDecl(n[g], (b, w // b, w // b), MATRIX), TensorDecl(n[g] + sfx, (b, w // b), BIAS)]
        return out + [TensorDecl(n["lambda"], (w,), BIAS), TensorDecl(n["o"], (h, w), MATRIX)]

    @staticmethod
    def _state_floats(spec) -> int:
        """Floats of the record in front of the convolution's rows: the state, rounded up to 4."""
        return -(-spec.width // 4) * 4

    @classmethod
    def cache_request(cls, spec):
        return FixedStateRequest((cls._state_floats(spec) + (spec.conv_taps - 1) * spec.width,))

    def load(self, store):
        s = self.spec
        n, sfx = self._names(s, self.prefix), s.bias_suffix
        self.w_in = pad_rows(store.cat([n["y"], n["x"]]))
        self.y_bias, self.x_bias = store.get(n["y"] + sfx), store.get(n["x"] + sfx)
        # [taps, channels]: a tap's weights of neighbouring channels are neighbours
        self.taps = store.get(n["conv"]).t().contiguous()
        self.conv_bias = store.get(n["conv"] + sfx)
        self.w_gates = torch.cat([store.get(n["r"]), store.get(n["i"])], dim=1).contiguous()      # [blocks, 2 n, n]
        self.r_bias, self.i_bias = (store.get(n[g] + sfx).reshape(-1).contiguous() for g in ("r", "i"))
        lam = store.get(n["lambda"]).to(torch.float64)
        self.rate = (-s.decay_coef * torch.nn.functional.softplus(lam)).to(torch.float32).contiguous()
        self.w_o = store.get(n["o"])

    def forward(self, ctx, x, cache, owns_cache):
        s = self.spec
        T = x.shape[0]
        proj = K.plain_unless(None, linear(x, self.w_in))              # [T, y | x]
        state = cache.state if cache.state.dim() == 2 else cache.state.view(cache.state.shape[0], -1)
        rows = state[:, self.state_floats:] if s.conv_taps > 1 else None
        u = torch.empty((T, s.width), dtype=x.dtype, device=x.device)
        K.short_conv(proj[:, s.width:], self.taps, rows, ctx, u, self.x_bias, self.conv_bias)
        z = block_diagonal_logits(u, self.w_gates)
        out = torch.empty_like(u)
        K.gated_recurrence(ctx, u, z, proj, state, out, r_bias=self.r_bias, i_bias=self.i_bias, rate=self.rate,
                           y_bias=self.y_bias)
        if self.out_dtype is not None:
            return linear(out, self.w_o, out_dtype=self.out_dtype)
        return linear(out, self.w_o, consumer="norm")
