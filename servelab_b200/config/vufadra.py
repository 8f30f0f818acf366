"""Typed configuration of the Vufadra decoder, read from its config.json keys.

A Vufadra model is a stack of layers that config.json lists one by one (``layers[i]``: ``type`` names
the mixer, ``mixer`` holds its sizes and constants, ``mlp`` the feed-forward or null).  Both sublayers
of a layer read the same stream, each behind a Dynamic Tanh norm of its own,
x <- x + mix(shift(N1(x))) + ff(N2(x)), where shift mixes a token's input with the previous token's.
``embedding.bigram`` = {buckets, mul_prev, mul_cur} adds a second embedding chosen by the token and
its predecessor.  ``loop`` = {start, stop, times}: the layers start .. stop - 1 run ``times`` times in
a row with the same weights, each pass with a cache and state of its own and each begun by
x <- W_in [x; x0] + step_t with the embedding output x0.  The output is the final norm and an untied
head.

Mixers: ``general_delta`` -- a delta rule with a decay and a removal rate per key channel; ``parallel``
-- two mixers on the same input, each result RMS-normed over the width, half their sum: ``left`` a
grouped-query attention over fixed chunks of ``mask.size`` positions whose weights are sigmoids of the
score plus a number a head, queries and keys normed a head and rotated (element i with element
i + dims / 2, ``rot.scaling`` = {factor, original, fast, slow}), ``right`` a linear attention with a
learned decay exp(-exp(z)), a bonus for the current token and inputs mixed with the previous token's;
``rglru`` -- a real-gated linear recurrence over ``width`` channels behind a convolution of ``conv``
taps, gates from ``blocks`` diagonal blocks.  Feed-forward ``dense``: down(silu(gate) up).

Any other key is an error: a key that is not read would be a mechanism that is not computed.

Tensor names: ``embed``, ``bigram``, ``loop.in``, ``loop.step``, ``final.norm``, ``head``, and under
``l<i>.``: ``norm1``, ``norm2`` (each with ``.b`` and ``.alpha``), ``shift``;
``mix.{r,k,v,g,a,a.b,w1,w2,w0,norm,o}``; ``mix.left.{q,k,v,o,q.norm,k.norm,pb}``,
``mix.right.{r,k,v,g,o,w1,w2,w0,u,norm}`` and ``mix.right.mu.{r,k,v,g,w}``, ``mix.left.out``,
``mix.right.out``; ``mix.{y,x,conv,ra,ri,lam,o}`` with ``.b`` biases; ``mlp.{gate,up,down}``.
"""

from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .daferax import _freeze, _only, _thaw
from .qwen2 import ConfigError
from .specs import (BigramSpec, BlockSpec, DecayAttentionSpec, DeltaRuleSpec, DynamicTanhSpec, GatedMLPSpec,
                    GatedRecurrenceSpec, LayerRun, LoopEntrySpec, ModelSpec, NoPositionSpec,
                    NormedAttentionSpec, ParallelMixersSpec, RotarySpec)

_MAX_POSITIONS = 1 << 20          # nothing in the model bounds the positions
DELTA_DECAY_COEF = math.exp(-0.5)  # decays of the delta rule: exp(-coef sigmoid(z))
UNIT_KEY_EPS = 1e-6               # u = k / sqrt(sum k^2 + eps)
RGLRU_COEF = 8.0                  # log a = -coef r softplus(lambda)
BRANCH_FACTOR = 0.5               # a parallel mixer returns half the sum of its two normed branches

_MIXER_TYPES = ("general_delta", "parallel", "rglru")


@dataclass(frozen=True)
class VufadraConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[dict, ...]               # the entries of config.json's ``layers``, frozen
    loop: Optional[Tuple[int, int, int]] = None      # (start, stop, times)
    bigram: Optional[Tuple[int, int, int]] = None    # (buckets, mul_prev, mul_cur)
    eos_token_ids: Tuple[int, ...] = ()

    architecture = "Vufadra"
    model_type = "vufadra"

    # ------------------------------------------------------------ parsing
    @classmethod
    def from_dict(cls, cfg: Dict[str, Any]) -> "VufadraConfig":
        p = []
        _only(cfg, ("architecture", "architectures", "model_type", "vocab", "width", "norm", "layers", "loop",
                    "embedding", "eos_token_id"), "config", p)
        for key in ("vocab", "width", "norm", "layers"):
            if key not in cfg:
                p.append(f"missing key '{key}'")
        if p:
            raise ConfigError("invalid Vufadra config: " + "; ".join(p))
        _only(cfg["norm"], ("eps",), "norm", p)
        loop = cfg.get("loop")
        if loop:
            _only(loop, ("start", "stop", "times"), "loop", p)
        embedding = cfg.get("embedding") or {}
        _only(embedding, ("bigram",), "embedding", p)
        bigram = embedding.get("bigram")
        if bigram:
            _only(bigram, ("buckets", "mul_prev", "mul_cur"), "embedding.bigram", p)
        if p:
            raise ConfigError("invalid Vufadra config: " + "; ".join(p))
        eos = cfg.get("eos_token_id", ())
        eos_ids = tuple(int(e) for e in eos) if isinstance(eos, (list, tuple)) else (int(eos),)
        try:
            out = cls(vocab=int(cfg["vocab"]), width=int(cfg["width"]), norm_eps=float(cfg["norm"]["eps"]),
                      layers=tuple(_freeze(layer) for layer in cfg["layers"]),
                      loop=(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None,
                      bigram=((int(bigram["buckets"]), int(bigram["mul_prev"]), int(bigram["mul_cur"]))
                              if bigram else None),
                      eos_token_ids=eos_ids)
        except (KeyError, TypeError, ValueError) as e:
            raise ConfigError(f"invalid Vufadra config: missing or malformed key {e}") from None
        out.to_model_spec()                # every per-layer check happens there
        return out

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
             "norm": {"eps": self.norm_eps}, "layers": [_thaw(layer) for layer in self.layers]}
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.bigram is not None:
            d["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), self.bigram))}
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    # ----------------------------------------------- the model as plain data
    def _attention(self, m: dict, where: str, p) -> NormedAttentionSpec:
        _only(m, ("heads", "kv_heads", "dim", "vdim", "mask", "rot", "scale"), where, p)
        heads, dim = int(m["heads"]), int(m["dim"])
        kv_heads, vdim = int(m.get("kv_heads", heads)), int(m.get("vdim", dim))
        if min(heads, kv_heads, dim, vdim) <= 0 or heads % kv_heads:
            p.append(f"{where}: heads must be a positive multiple of kv_heads; dim and vdim positive")
        mask, chunk = m.get("mask"), None
        if mask:
            _only(mask, ("size",), where + ".mask", p)
            chunk = int(mask["size"])
            if chunk < 1:
                p.append(f"{where}.mask.size must be at least 1")
        position, rot = NoPositionSpec(), m.get("rot")
        if rot:
            _only(rot, ("base", "dims", "scaling"), where + ".rot", p)
            dims = int(rot["dims"])
            if dims % 2 or not 0 < dims <= dim:
                p.append(f"{where}.rot.dims must be even, positive and at most dim")
            sc, yarn = rot.get("scaling"), {}
            if sc:
                _only(sc, ("factor", "original", "fast", "slow"), where + ".rot.scaling", p)
                yarn = dict(yarn_factor=float(sc["factor"]), yarn_original=float(sc["original"]),
                            yarn_fast=float(sc["fast"]), yarn_slow=float(sc["slow"]))
                if min(yarn.values()) <= 0:
                    p.append(f"{where}.rot.scaling: factor, original, fast and slow must be positive")
            position = RotarySpec(head_dim=dim, rotary_dim=dims, theta=float(rot["base"]), precise=True, **yarn)
        return NormedAttentionSpec(
            hidden_size=self.width, num_heads=heads, num_kv_heads=kv_heads, head_dim=dim, value_dim=vdim,
            chunk=chunk, scale=float(m["scale"]), qk_norm=True, qk_norm_eps=self.norm_eps, position=position,
            weight_fn="sigmoid", score_bias=True)

    # (``rank``, the bottleneck of a decay's projection, is optional: a checkpoint's w1 decides it)
    def _time_mix(self, m: dict, where: str, p) -> DecayAttentionSpec:
        _only(m, ("heads", "dim", "rank"), where, p)
        heads, dim = int(m["heads"]), int(m["dim"])
        if min(heads, dim) <= 0:
            p.append(f"{where}: heads and dim must be positive")
        return DecayAttentionSpec(
            hidden_size=self.width, num_heads=heads, head_dim=dim, value_dim=dim, decay=(), out_norm="head",
            out_norm_weight=True, out_norm_eps=self.norm_eps, gate_activation="silu",
            decay_gate_rank=int(m.get("rank", -1)), decay_gate_kind="exp_exp", decay_gate_tanh=True, bonus=True,
            token_mix=True, q_name="r", decay_down_name="w1", decay_up_name="w2", decay_bias_name="w0")

    def _mixer(self, i: int, kind: str, m: dict, p):
        where = f"layers[{i}].mixer"
        if kind == "general_delta":
            _only(m, ("heads", "dim", "rank"), where, p)
            heads, dim = int(m["heads"]), int(m["dim"])
            if min(heads, dim) <= 0:
                p.append(f"{where}: heads and dim must be positive")
            return DeltaRuleSpec(hidden_size=self.width, num_heads=heads, head_dim=dim, value_dim=dim,
                                 decay_coef=DELTA_DECAY_COEF, decay_rank=int(m.get("rank", -1)),
                                 unit_eps=UNIT_KEY_EPS, out_norm_eps=self.norm_eps)
        if kind == "rglru":
            _only(m, ("width", "blocks", "conv"), where, p)
            width, blocks, taps = int(m["width"]), int(m["blocks"]), int(m["conv"])
            if min(width, blocks, taps) <= 0 or width % blocks:
                p.append(f"{where}: width must be a positive multiple of blocks, conv at least 1")
            return GatedRecurrenceSpec(hidden_size=self.width, width=width, blocks=blocks, conv_taps=taps,
                                       decay_coef=RGLRU_COEF)
        _only(m, ("left", "right"), where, p)
        return ParallelMixersSpec(
            hidden_size=self.width, left=self._attention(m["left"], where + ".left", p),
            right=self._time_mix(m["right"], where + ".right", p), eps=self.norm_eps, factor=BRANCH_FACTOR)

    def _feed_forward(self, i: int, mlp: dict, p):
        where = f"layers[{i}].mlp"
        kind = mlp.get("kind", "dense")
        if kind != "dense":
            p.append(f"{where}: kind {kind!r} is not known (dense)")
            return None
        _only(mlp, ("kind", "ff"), where, p)
        if int(mlp["ff"]) <= 0:
            p.append(f"{where}.ff must be positive")
        return GatedMLPSpec(hidden_size=self.width, intermediate_size=int(mlp["ff"]), activation="silu",
                            gate_name="gate", up_name="up", down_name="down", weight_suffix="")

    def run_order(self) -> Tuple[LayerRun, ...]:
        """The layers in the order they run, a looped layer once per pass."""
        n = len(self.layers)
        if self.loop is None:
            return tuple(LayerRun(i) for i in range(n))
        start, stop, times = self.loop
        runs = [LayerRun(i) for i in range(start)]
        for t in range(times):
            runs += [LayerRun(i, loop_entry=t if i == start else None) for i in range(start, stop)]
        return tuple(runs + [LayerRun(i) for i in range(stop, n)])

    def to_model_spec(self) -> ModelSpec:
        p = []
        if self.vocab <= 0 or self.width <= 0:
            p.append("vocab and width must be positive")
        if not self.layers:
            p.append("the model has no layers")
        if self.loop is not None:
            start, stop, times = self.loop
            if not 0 <= start < stop <= len(self.layers) or times < 1:
                p.append("loop: 0 <= start < stop <= number of layers and times >= 1 are needed")
        if self.bigram is not None and self.bigram[0] < 1:
            p.append("embedding.bigram.buckets must be at least 1")
        norm = DynamicTanhSpec(dim=self.width, weight_suffix="", bias_suffix=".b", alpha_suffix=".alpha")
        layers = []
        for i, entry in enumerate(_thaw(layer) for layer in self.layers):
            _only(entry, ("type", "mixer", "mlp"), f"layers[{i}]", p)
            kind = entry.get("type")
            if kind not in _MIXER_TYPES:
                p.append(f"layers[{i}]: mixer type {kind!r} is not known ({', '.join(_MIXER_TYPES)})")
                continue
            try:
                mixer = self._mixer(i, kind, entry.get("mixer") or {}, p)
                ff = self._feed_forward(i, entry["mlp"], p) if entry.get("mlp") else None
            except (KeyError, TypeError, ValueError) as e:
                p.append(f"layers[{i}]: missing or malformed key {e}")
                continue
            layers.append(BlockSpec(kind="parallel_norm", mixer=mixer, feed_forward=ff, mixer_norm=norm,
                                    ff_norm=None if ff is None else norm, mixer_norm_name="norm1",
                                    mixer_name="mix", ff_norm_name="norm2", feed_forward_name="mlp",
                                    token_shift=True, shift_name="shift"))
        if p:
            raise ConfigError("invalid Vufadra config: " + "; ".join(p))
        return ModelSpec(
            architecture=self.architecture, hidden_size=self.width, vocab_size=self.vocab,
            layers=tuple(layers), run_order=self.run_order(), final_norm=norm,
            tie_word_embeddings=False, max_position_embeddings=_MAX_POSITIONS, eos_token_ids=self.eos_token_ids,
            embed_name="embed", lm_head_name="head", final_norm_prefix="final.norm", layer_prefix="l{}",
            bigram=None if self.bigram is None else BigramSpec(*self.bigram),
            loop=None if self.loop is None else LoopEntrySpec(times=self.loop[2]),
            # a layer without a feed-forward has no use for its second norm; a checkpoint may hold it
            ignored_suffixes=(".norm2", ".norm2.b", ".norm2.alpha"))
