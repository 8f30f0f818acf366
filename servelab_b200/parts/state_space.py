"""A selective state space with a short convolution and a gated norm (spec: ``StateSpaceSpec``).

Per step, with h the mixer's input [T, hidden]:

  1. one product for z | x | B | C; the step sizes' logits dt by a product of their own with float32
     results (they enter the recurrence's exponentials);
  2. the causal convolution of the x | B | C channels with its bias, and SiLU; a request's last
     ``conv_taps`` - 1 rows are part of its record;
  3. the recurrence over the tokens of every request in order -- step sizes, decays and the state in
     float32; the state lives in the request's slot and is carried from step to step, so a prompt may be
     cut anywhere;
  4. one kernel: times silu(z), every part of the row divided by its root mean square, the weight;
  5. the output projection.
"""

from __future__ import annotations

import torch

from ..cache.manager import FixedStateRequest
from ..ops import kernels as K
from ..ops.linear import linear, narrow_logits, narrow_logits_by_library
from ..weights.source import BIAS, MATRIX, NORM, TensorDecl
from .base import Mixer
from .normed_attention import pad_rows
from .registry import register_mixer

MAX_STATE_DIM = 256


@register_mixer("state_space")
class StateSpace(Mixer):
    graph_safe = True
    splits_projections = True
    padded_steps_safe = True      # requests without tokens and tokens of no request leave the records alone

    def __init__(self, spec, prefix, env):
        super().__init__(spec, prefix, env)
        s = spec
        if min(s.num_heads, s.value_dim, s.state_dim, s.groups, s.norm_groups) <= 0 or s.num_heads % s.groups:
            raise ValueError("state_space: sizes must be positive and heads a multiple of groups")
        if s.state_dim > MAX_STATE_DIM:
            raise ValueError(f"state_space: at most {MAX_STATE_DIM} state elements, got {s.state_dim}")
        self.inner = s.num_heads * s.value_dim
        if self.inner % s.norm_groups:
            raise ValueError("state_space: norm_groups must divide heads * value_dim")
        if not 1 <= s.conv_taps <= K.CONV_MAX_TAPS:
            raise ValueError(f"state_space: 1..{K.CONV_MAX_TAPS} taps, got {s.conv_taps}")
        self.channels = self._channels(s)
        self.state_floats = self._state_floats(s)
        self.out_width = self.inner
        self.out_dtype = None                  # (set by a mixer that wraps this one)
        self.o_bias = None

    @staticmethod
    def _channels(spec) -> int:
        """Channels of the convolution: x | B | C."""
        return spec.num_heads * spec.value_dim + 2 * spec.groups * spec.state_dim

    @staticmethod
    def _state_floats(spec) -> int:
        """Floats of the record in front of the convolution's rows: the state, rounded up to 4."""
        return -(-spec.num_heads * spec.state_dim * spec.value_dim // 4) * 4

    @classmethod
    def _names(cls, spec, prefix):
        return {n: f"{prefix}.{getattr(spec, n + '_name')}"
                for n in ("in", "conv", "conv_bias", "dt_bias", "decay", "skip", "norm", "o")}

    @classmethod
    def declare(cls, spec, prefix):
        h, H, inner, C = spec.hidden_size, spec.num_heads, spec.num_heads * spec.value_dim, cls._channels(spec)
        n = cls._names(spec, prefix)
        return [TensorDecl(n["in"], (inner + C + H, h), MATRIX), TensorDecl(n["conv"], (C, spec.conv_taps), BIAS),
                TensorDecl(n["conv_bias"], (C,), BIAS), TensorDecl(n["dt_bias"], (H,), BIAS),
                TensorDecl(n["decay"], (H,), BIAS), TensorDecl(n["skip"], (H,), BIAS),
                TensorDecl(n["norm"], (inner,), NORM), TensorDecl(n["o"], (h, inner), MATRIX)]

    @classmethod
    def cache_request(cls, spec):
        return FixedStateRequest((cls._state_floats(spec) + (spec.conv_taps - 1) * cls._channels(spec),))

    def load(self, store):
        s = self.spec
        n = self._names(s, self.prefix)
        w = store.get(n["in"])
        split = self.inner + self.channels
        self.w_in = pad_rows(w[:split].contiguous())
        self.w_dt = pad_rows(w[split:].contiguous())
        self.w_dt_f32 = w[split:].to(torch.float32).contiguous()
        # [taps, channels]: a tap's weights of neighbouring channels are neighbours
        self.taps = store.get(n["conv"]).t().contiguous()
        self.conv_bias = store.get(n["conv_bias"])
        self.dt_bias, self.skip = store.get(n["dt_bias"]), store.get(n["skip"])
        self.rate = torch.exp(store.get(n["decay"]).to(torch.float64)).to(torch.float32).contiguous()
        self.norm_w = store.get(n["norm"])
        self.w_o = store.get(n["o"])

    def forward(self, ctx, x, cache, owns_cache):
        proj = K.plain_unless(None, linear(x, self.w_in))              # [T, z | x | B | C]
        out = torch.empty((x.shape[0], self.inner), dtype=x.dtype, device=x.device)
        self.core(ctx, x, proj, cache, owns_cache, out)
        if self.out_dtype is not None:
            return linear(out, self.w_o, out_dtype=self.out_dtype)
        return linear(out, self.w_o, consumer="norm")

    def early(self, ctx, x):
        """The step sizes' logits, where they come from a product of the library."""
        return narrow_logits(x, self.w_dt, self.w_dt_f32) if narrow_logits_by_library(x) else None

    def core(self, ctx, x, proj, cache, owns_cache, out, factor=1.0, early=None):
        s = self.spec
        T = x.shape[0]
        if not owns_cache:
            raise NotImplementedError("state_space: a run that reads another run's cache")
        dt = narrow_logits(x, self.w_dt, self.w_dt_f32) if early is None else early
        state = cache.state if cache.state.dim() == 2 else cache.state.view(cache.state.shape[0], -1)
        rows = state[:, self.state_floats:] if s.conv_taps > 1 else None
        u = torch.empty((T, self.channels), dtype=x.dtype, device=x.device)
        K.short_conv(proj[:, self.inner:], self.taps, rows, ctx, u, None, self.conv_bias, activation="silu")
        y = torch.empty((T, self.inner), dtype=torch.float32, device=x.device)
        K.state_space(ctx, u, dt, state, y, num_heads=s.num_heads, value_dim=s.value_dim, state_dim=s.state_dim,
                      groups=s.groups, dt_bias=self.dt_bias, rate=self.rate, skip=self.skip)
        K.gate_group_norm(y, proj, s.norm_groups, out, eps=s.norm_eps, weight=self.norm_w, factor=factor)
