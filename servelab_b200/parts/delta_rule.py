"""Linear attention by a delta rule with a decay and a removal rate per key channel (spec:
``DeltaRuleSpec``).

Per step, with h the mixer's input [T, hidden]:

  1. one product for r | k | v | gate | removal | the decays' bottleneck (concatenated at load);
  2. the bottleneck's second product behind a tanh, float32 results;
  3. the recurrence over the tokens of every request in order -- unit keys, decays, removal rates and
     the state in float32; the state lives in the request's slot and is carried from step to step, so a
     prompt may be cut anywhere -- then the head norm, the row's weight and sigmoid(gate) (in the same
     launch token by token; in chunks, one more);
  4. the output projection.
"""

from __future__ import annotations

import torch

from ..cache.manager import FixedStateRequest
from ..ops import kernels as K
from ..ops.linear import linear
from ..weights.source import BIAS, MATRIX, NORM, TensorDecl
from .base import Mixer
from .normed_attention import pad_rows
from .registry import register_mixer

MAX_HEAD_DIM = 256


@register_mixer("delta_rule")
class DeltaRule(Mixer):
    graph_safe = True
    padded_steps_safe = True      # requests without tokens and tokens of no request leave the records alone

    def __init__(self, spec, prefix, env):
        super().__init__(spec, prefix, env)
        s = spec
        if min(s.num_heads, s.head_dim, s.value_dim) <= 0 or s.head_dim > MAX_HEAD_DIM:
            raise ValueError(f"delta_rule: heads, head_dim (at most {MAX_HEAD_DIM}) and value_dim must be positive")
        if s.decay_coef < 0:
            raise ValueError("delta_rule: decay_coef must not be negative")
        self.out_dtype = None                  # (set by a mixer that wraps this one)
        self.q_size = s.num_heads * s.head_dim
        self.v_size = s.num_heads * s.value_dim

    @classmethod
    def _names(cls, spec, prefix):
        return {n: f"{prefix}.{getattr(spec, n + '_name')}"
                for n in ("r", "k", "v", "gate", "o", "removal", "removal_bias", "decay_down", "decay_up",
                          "decay_bias", "out_norm")}

    @classmethod
    def declare(cls, spec, prefix):
        h, qs, vs = spec.hidden_size, spec.num_heads * spec.head_dim, spec.num_heads * spec.value_dim
        r = spec.decay_rank                     # (-1: the checkpoint's tensor decides)
        n = cls._names(spec, prefix)
        return [TensorDecl(n["r"], (qs, h), MATRIX), TensorDecl(n["k"], (qs, h), MATRIX),
                TensorDecl(n["v"], (vs, h), MATRIX), TensorDecl(n["gate"], (vs, h), MATRIX),
                TensorDecl(n["removal"], (qs, h), MATRIX), TensorDecl(n["removal_bias"], (qs,), BIAS),
                TensorDecl(n["decay_down"], (r, h), MATRIX), TensorDecl(n["decay_up"], (qs, r), MATRIX),
                TensorDecl(n["decay_bias"], (qs,), BIAS), TensorDecl(n["out_norm"], (vs,), NORM),
                TensorDecl(n["o"], (h, vs), MATRIX)]

    @classmethod
    def cache_request(cls, spec):
        return FixedStateRequest((spec.num_heads, spec.head_dim, spec.value_dim))

    def load(self, store):
        n = self._names(self.spec, self.prefix)
        self.w_in = pad_rows(store.cat([n["r"], n["k"], n["v"], n["gate"], n["removal"], n["decay_down"]]))
        self.rank = store.get(n["decay_down"]).shape[0]
        self.w_up = store.get(n["decay_up"])
        self.decay_bias = store.get(n["decay_bias"])
        self.removal_bias = store.get(n["removal_bias"])
        self.norm_w = store.get(n["out_norm"])
        self.w_o = store.get(n["o"])

    def forward(self, ctx, x, cache, owns_cache):
        s = self.spec
        T = x.shape[0]
        proj = K.plain_unless(None, linear(x, self.w_in))
        g_off = 2 * self.q_size + self.v_size
        a_off = g_off + self.v_size
        low = proj[:, a_off + self.q_size:a_off + self.q_size + self.rank]
        gate_z = torch.empty((T, self.q_size), dtype=torch.float32, device=x.device)
        K.tanh_linear(low, self.w_up, self.decay_bias, gate_z)
        state = cache.state if cache.state.dim() == 2 else cache.state.view(cache.state.shape[0], -1)
        out = torch.empty((T, self.v_size), dtype=x.dtype, device=x.device)
        K.delta_rule(ctx, proj, state, out, r_off=0, k_off=self.q_size, v_off=2 * self.q_size, a_off=a_off,
                     g_off=g_off, num_heads=s.num_heads, head_dim=s.head_dim, value_dim=s.value_dim,
                     a_bias=self.removal_bias, gate_z=gate_z, decay_coef=s.decay_coef, unit_eps=s.unit_eps,
                     norm_w=self.norm_w, norm_eps=s.out_norm_eps)
        if self.out_dtype is not None:
            return linear(out, self.w_o, out_dtype=self.out_dtype)
        return linear(out, self.w_o, consumer="norm")
