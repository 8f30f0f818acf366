"""Typed configuration of the Sunutar decoder, read from its config.json keys.

A Sunutar model is a stack of layers that config.json lists one by one (``layers[i]``: ``type`` names the
mixer, ``mixer`` holds its sizes and constants, ``mlp`` the feed-forward or null).  A layer norms what a
sublayer reads and what it returns: x <- x + m N1b(mix(N1(x))), then x <- x + m N2b(ff(N2(x))) with RMS
norms and m = ``residual_mult``.  The output is the final norm and the embedding table.

Mixer ``parallel``: ``left_scale`` times a left branch plus ``right_scale`` times a right one, both on the same
input.  Left: grouped-query softmax attention with biases on q, k, v and the output, q and k RMS-normed
over the whole projected rows, no rotation; a score times ``scale`` is soft-capped by ``softcap``, then
slope_h (i - j) is taken off with slope_h = 2^(-8 (h + 1) / heads); a sliding window ``mask.size``; one is
added to the softmax's denominator.  Right: a selective state space of ``heads`` heads with values of
``vdim`` and a state of ``state`` elements, B and C shared by the heads of a group (``groups``), a causal
convolution of ``conv`` taps on x, B and C, the result gated by SiLU and then normed in ``norm_groups`` parts.
Feed-forward ``dense``: g = min(gate, limit), u = clamp(up, -limit, limit), down(g sigmoid(1.702 g) (u + 1));
``moe``: ``router.experts`` such feed-forwards of ``expert.ff`` elements, of which a token uses the
``router.top`` with the largest sigmoid scores; an expert's input is its score times the token's.

Any other key is an error: a key that is not read would be a mechanism that is not computed.

Tensor names: ``embed``, ``final.norm``, and under ``l<i>.``: ``norm1``, ``norm1b``, ``norm2``, ``norm2b``;
``mix.left.{q,k,v,o}`` with ``.b`` biases, ``mix.left.{q.norm,k.norm}``;
``mix.right.{in,conv,conv.b,dt_bias,A_log,D,norm,o}``; ``mlp.{gate,up,down}`` or ``mlp.router`` and
``mlp.e<j>.{gate,up,down}``.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Tuple

from .daferax import _freeze, _only, _thaw
from .qwen2 import ConfigError
from .specs import (BlockSpec, GatedMLPSpec, LayerRun, ModelSpec, NormedAttentionSpec, ParallelMixersSpec,
                    RMSNormSpec, RoutedExpertsSpec, StateSpaceSpec)
from .sumolorn import SWISH_ALPHA, _window

_MAX_POSITIONS = 1 << 20          # nothing in the model bounds the positions
SLOPE_SPAN = 8.0                  # slope_h = 2^(-span (h + 1) / heads)
SINK_SCORE = 0.0                  # the score whose exponential joins every denominator: one is added

_MIXER_TYPES = ("parallel",)


@dataclass(frozen=True)
class SunutarConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[dict, ...]               # the entries of config.json's ``layers``, frozen
    residual_mult: float = 1.0
    eos_token_ids: Tuple[int, ...] = ()

    architecture = "Sunutar"
    model_type = "sunutar"

    # ------------------------------------------------------------ parsing
    @classmethod
    def from_dict(cls, cfg: Dict[str, Any]) -> "SunutarConfig":
        p = []
        _only(cfg, ("architecture", "architectures", "model_type", "vocab", "width", "norm", "layers",
                    "residual_mult", "eos_token_id"), "config", p)
        for key in ("vocab", "width", "norm", "layers"):
            if key not in cfg:
                p.append(f"missing key '{key}'")
        if p:
            raise ConfigError("invalid Sunutar config: " + "; ".join(p))
        _only(cfg["norm"], ("eps",), "norm", p)
        if p:
            raise ConfigError("invalid Sunutar config: " + "; ".join(p))
        eos = cfg.get("eos_token_id", ())
        eos_ids = tuple(int(e) for e in eos) if isinstance(eos, (list, tuple)) else (int(eos),)
        try:
            out = cls(vocab=int(cfg["vocab"]), width=int(cfg["width"]), norm_eps=float(cfg["norm"]["eps"]),
                      layers=tuple(_freeze(layer) for layer in cfg["layers"]),
                      residual_mult=float(cfg.get("residual_mult", 1.0)), eos_token_ids=eos_ids)
        except (KeyError, TypeError, ValueError) as e:
            raise ConfigError(f"invalid Sunutar config: missing or malformed key {e}") from None
        out.to_model_spec()                # every per-layer check happens there
        return out

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
             "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult,
             "layers": [_thaw(layer) for layer in self.layers]}
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    # ----------------------------------------------- the model as plain data
    def _attention(self, m: dict, where: str, p) -> NormedAttentionSpec:
        _only(m, ("heads", "kv_heads", "dim", "vdim", "mask", "scale", "softcap"), where, p)
        heads, dim = int(m["heads"]), int(m["dim"])
        kv_heads, vdim = int(m.get("kv_heads", heads)), int(m.get("vdim", dim))
        if min(heads, kv_heads, dim, vdim) <= 0 or heads % kv_heads:
            p.append(f"{where}: heads must be a positive multiple of kv_heads; dim and vdim positive")
        cap = m.get("softcap")
        if float(m["scale"]) <= 0 or (cap is not None and float(cap) <= 0):
            p.append(f"{where}: scale and softcap must be positive")
        return NormedAttentionSpec(
            hidden_size=self.width, num_heads=heads, num_kv_heads=kv_heads, head_dim=dim, value_dim=vdim,
            window=_window(m, where, p), scale=float(m["scale"]), qk_row_norm=True, qk_norm_eps=self.norm_eps,
            qkv_bias=True, out_bias=True, softcap=None if cap is None else float(cap), sink_score=SINK_SCORE,
            distance_slopes=tuple(2.0 ** (-SLOPE_SPAN * (h + 1) / heads) for h in range(heads)))

    def _state_space(self, m: dict, where: str, p) -> StateSpaceSpec:
        _only(m, ("heads", "vdim", "state", "groups", "conv", "norm_groups"), where, p)
        heads, vdim, state, groups, conv, norm_groups = (
            int(m[k]) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups"))
        if min(heads, vdim, state, groups, conv, norm_groups) <= 0 or heads % groups or (heads * vdim) % norm_groups:
            p.append(f"{where}: sizes must be positive, heads a multiple of groups and heads * vdim of norm_groups")
        return StateSpaceSpec(hidden_size=self.width, num_heads=heads, value_dim=vdim, state_dim=state, groups=groups,
                              conv_taps=conv, norm_groups=norm_groups, norm_eps=self.norm_eps)

    def _mixer(self, i: int, m: dict, p) -> ParallelMixersSpec:
        where = f"layers[{i}].mixer"
        _only(m, ("left", "right", "left_scale", "right_scale"), where, p)
        return ParallelMixersSpec(
            hidden_size=self.width, left=self._attention(m["left"], where + ".left", p),
            right=self._state_space(m["right"], where + ".right", p), branch_norms=False,
            left_factor=float(m.get("left_scale", 1.0)), right_factor=float(m.get("right_scale", 1.0)))

    def _feed_forward(self, i: int, mlp: dict, p):
        where = f"layers[{i}].mlp"
        kind = mlp.get("kind", "dense")
        if kind == "dense":
            _only(mlp, ("kind", "ff", "limit"), where, p)
            if int(mlp["ff"]) <= 0 or float(mlp["limit"]) <= 0:
                p.append(f"{where}: ff and limit must be positive")
            return GatedMLPSpec(hidden_size=self.width, intermediate_size=int(mlp["ff"]), activation="swish_clamped",
                                limit=float(mlp["limit"]), swish_alpha=SWISH_ALPHA, gate_name="gate", up_name="up",
                                down_name="down", weight_suffix="")
        if kind != "moe":
            p.append(f"{where}: kind {kind!r} is not known (dense, moe)")
            return None
        _only(mlp, ("kind", "expert", "router"), where, p)
        _only(mlp["expert"], ("ff", "limit"), where + ".expert", p)
        _only(mlp["router"], ("experts", "top"), where + ".router", p)
        experts, top, ff = int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"])
        if not 0 < top <= experts or ff <= 0 or float(mlp["expert"]["limit"]) <= 0:
            p.append(f"{where}: 0 < router.top <= router.experts; expert.ff and expert.limit positive")
        return RoutedExpertsSpec(
            hidden_size=self.width, num_experts=experts, top=top, expert_size=ff, score_fn="sigmoid",
            activation="swish_clamped", limit=float(mlp["expert"]["limit"]), swish_alpha=SWISH_ALPHA,
            weight_inputs=True)

    def to_model_spec(self) -> ModelSpec:
        p = []
        if self.vocab <= 0 or self.width <= 0:
            p.append("vocab and width must be positive")
        if not self.layers:
            p.append("the model has no layers")
        norm = RMSNormSpec(dim=self.width, eps=self.norm_eps, weight_suffix="")
        after = RMSNormSpec(dim=self.width, eps=self.norm_eps, weight_suffix="", factor=self.residual_mult)
        layers = []
        for i, entry in enumerate(_thaw(layer) for layer in self.layers):
            _only(entry, ("type", "mixer", "mlp"), f"layers[{i}]", p)
            kind = entry.get("type")
            if kind not in _MIXER_TYPES:
                p.append(f"layers[{i}]: mixer type {kind!r} is not known ({', '.join(_MIXER_TYPES)})")
                continue
            try:
                mixer = self._mixer(i, entry.get("mixer") or {}, p)
                ff = self._feed_forward(i, entry["mlp"], p) if entry.get("mlp") else None
            except (KeyError, TypeError, ValueError) as e:
                p.append(f"layers[{i}]: missing or malformed key {e}")
                continue
            layers.append(BlockSpec(kind="sandwich_norm", mixer=mixer, feed_forward=ff, mixer_norm=norm,
                                    mixer_post_norm=after, ff_norm=None if ff is None else norm,
                                    ff_post_norm=None if ff is None else after, mixer_norm_name="norm1",
                                    mixer_name="mix", ff_norm_name="norm2", feed_forward_name="mlp",
                                    mixer_post_norm_name="norm1b", ff_post_norm_name="norm2b"))
        if p:
            raise ConfigError("invalid Sunutar config: " + "; ".join(p))
        return ModelSpec(
            architecture=self.architecture, hidden_size=self.width, vocab_size=self.vocab,
            layers=tuple(layers), run_order=tuple(LayerRun(i) for i in range(len(layers))), final_norm=norm,
            tie_word_embeddings=True, max_position_embeddings=_MAX_POSITIONS, eos_token_ids=self.eos_token_ids,
            embed_name="embed", lm_head_name="head", final_norm_prefix="final.norm", layer_prefix="l{}",
            # a layer without a feed-forward has no use for its second norms; a checkpoint may hold them
            ignored_suffixes=(".norm2", ".norm2b"))
