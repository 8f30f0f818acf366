"""Sunutar on the CPU: config keys and refusals, the spec it turns into, the tensors it declares, what its
blocks ask of the cache, the merged matrices of a parallel mixer, and the oracle's own pieces on cases worked
by hand."""

import copy
import json
import math

import pytest
import torch

import plain_sunutar as plain
import sunutar_cases as C
from servelab_b200.cache.manager import paged_part, record_floats
from servelab_b200.config import ConfigError, SunutarConfig, config_from_dict, load_config
from servelab_b200.config.specs import NormedAttentionSpec, ParallelMixersSpec, RMSNormSpec, StateSpaceSpec
from servelab_b200.models.causal_lm import CausalLM, declare_tensors
from servelab_b200.parts import BLOCKS, BuildEnv, part_class
from servelab_b200.parts.normed_attention import NormedAttention
from servelab_b200.parts.parallel_mixers import ParallelMixers
from servelab_b200.parts.routed_experts import RoutedExperts
from servelab_b200.parts.state_space import StateSpace
from servelab_b200.weights import RandomSource

F64 = torch.float64
CPU = BuildEnv(device="cpu", dtype=torch.float32)


def test_round_trip_and_registry(tmp_path):
    for cfg, _, _ in C.CASES.values():
        typed = config_from_dict(cfg)
        assert isinstance(typed, SunutarConfig) and typed.to_dict() == cfg
        assert hash(typed) == hash(config_from_dict(copy.deepcopy(cfg)))
    with open(tmp_path / "config.json", "w") as f:
        json.dump(C.A, f)
    assert load_config(str(tmp_path)).to_dict() == C.A


def test_every_size_and_constant_reaches_the_spec():
    spec = config_from_dict(C.A).to_model_spec()
    assert spec.vocab_size == 211 and spec.hidden_size == 48 and spec.tie_word_embeddings
    assert spec.final_norm.kind == "rmsnorm" and spec.final_norm.factor == 1.0 and not spec.final_norm.unit_offset
    assert [r.layer for r in spec.run_order] == [0, 1, 2]
    for b in spec.layers:
        assert b.kind == "sandwich_norm" and b.mixer_norm.factor == 1.0 and b.mixer_post_norm.factor == 0.55
        assert b.mixer_norm.eps == b.mixer_post_norm.eps == 1e-6
    assert spec.layers[1].feed_forward is None and spec.layers[1].ff_post_norm is None
    assert spec.layers[2].ff_post_norm.factor == 0.55
    par = spec.layers[0].mixer
    assert (par.branch_norms, par.left_factor, par.right_factor) == (False, 0.6, 1.1)
    lf, rt = par.left, par.right
    assert (lf.num_heads, lf.num_kv_heads, lf.head_dim, lf.value_dim, lf.scale, lf.window, lf.softcap) == \
        (4, 2, 16, 8, 0.4, 5, 6.0)
    assert lf.qk_row_norm and not lf.qk_norm and lf.qkv_bias and lf.out_bias and lf.qk_norm_eps == 1e-6
    assert lf.sink_score == 0.0 and not lf.sink and lf.position.kind == "none"
    assert lf.distance_slopes == (2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8)
    six = spec.layers[1].mixer.left.distance_slopes
    assert len(six) == 6 and all(abs(s - 2 ** (-8 * (h + 1) / 6)) < 1e-15 for h, s in enumerate(six))
    assert (rt.num_heads, rt.value_dim, rt.state_dim, rt.groups, rt.conv_taps, rt.norm_groups, rt.norm_eps) == \
        (3, 16, 8, 1, 3, 4, 1e-6)
    assert spec.layers[2].mixer.left.window is None
    ff = spec.layers[0].feed_forward
    assert (ff.kind, ff.num_experts, ff.top, ff.expert_size, ff.limit, ff.activation, ff.swish_alpha) == \
        ("routed_experts", 5, 2, 24, 1.5, "swish_clamped", 1.702)
    assert ff.weight_inputs and not ff.renormalize and ff.score_fn == "sigmoid" and ff.route_scale == 1.0
    assert ff.correction_name is None and ff.shared is None and ff.num_groups == 1
    ff = spec.layers[2].feed_forward
    assert (ff.kind, ff.intermediate_size, ff.limit, ff.activation, ff.swish_alpha) == \
        ("gated_mlp", 40, 0.9, "swish_clamped", 1.702)
    assert config_from_dict(C.B).to_model_spec().layers[2].mixer.left.softcap is None
    assert config_from_dict(C.B).to_model_spec().layers[0].mixer_post_norm.factor == 1.0


@pytest.mark.parametrize("change", [
    lambda c: c.pop("width"), lambda c: c.update(rope=1), lambda c: c["norm"].update(kind="x"),
    lambda c: c["layers"][0].update(type="attention"), lambda c: c["layers"][0].update(extra=1),
    lambda c: c["layers"][0]["mixer"].update(middle={}), lambda c: c["layers"][0]["mixer"].pop("left"),
    lambda c: c["layers"][0]["mixer"]["left"].update(rot={"base": 1e4, "dims": 4}),
    lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), lambda c: c["layers"][0]["mixer"]["left"].pop("scale"),
    lambda c: c["layers"][0]["mixer"]["left"].update(softcap=0.0),
    lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(kind="chunk"),
    lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0),
    lambda c: c["layers"][0]["mixer"]["right"].update(groups=2), lambda c: c["layers"][0]["mixer"]["right"].pop("state"),
    lambda c: c["layers"][0]["mixer"]["right"].update(norm_groups=5), lambda c: c["layers"][0]["mixer"]["right"].update(conv=0),
    lambda c: c["layers"][0]["mixer"]["right"].update(clamp=1), lambda c: c["layers"][0]["mlp"].update(kind="glu"),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=6), lambda c: c["layers"][0]["mlp"]["router"].update(scale=1.0),
    lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), lambda c: c["layers"][2]["mlp"].update(limit=-1.0),
    lambda c: c["layers"][2]["mlp"].update(bias=True), lambda c: c.update(layers=[]),
])
def test_refusals(change):
    cfg = copy.deepcopy(C.A)
    change(cfg)
    with pytest.raises(ConfigError):
        config_from_dict(cfg)


def test_parts_refuse_what_is_not_built():
    att = dict(hidden_size=16, num_heads=2, num_kv_heads=1, head_dim=8, value_dim=8)
    for bad in (dict(qk_row_norm=True, qk_norm=True), dict(qkv_bias=True, conv_taps=2), dict(distance_slopes=(0.5,)),
                dict(sink=True, sink_score=0.0), dict(sink_score=0.0, weight_fn="sigmoid")):
        with pytest.raises(ValueError):
            NormedAttention(NormedAttentionSpec(**att, **bad), "x", CPU)
    ss = dict(hidden_size=16, num_heads=2, value_dim=8, state_dim=8)
    for bad in (dict(groups=3), dict(state_dim=300), dict(norm_groups=3), dict(conv_taps=0)):
        with pytest.raises(ValueError):
            StateSpace(StateSpaceSpec(**{**ss, **bad}), "x", CPU)
    ff = config_from_dict(C.A).to_model_spec().layers[0].feed_forward
    from dataclasses import replace
    for bad in (dict(limit=None), dict(activation="relu")):
        with pytest.raises(ValueError):
            RoutedExperts(replace(ff, **bad), "x", CPU)
    from servelab_b200.config.specs import DecayAttentionSpec
    decay = DecayAttentionSpec(hidden_size=16, num_heads=2, head_dim=8, value_dim=8, decay=(0.5, 0.9))
    with pytest.raises(ValueError, match="projections"):
        ParallelMixers(ParallelMixersSpec(hidden_size=16, left=NormedAttentionSpec(**att), right=decay,
                                          branch_norms=False), "x", CPU)


def test_declared_tensors():
    d = {t.name: tuple(t.shape) for t in declare_tensors(config_from_dict(C.A).to_model_spec())}
    assert d["embed"] == (211, 48) and d["final.norm"] == (48,) and "head" not in d
    assert d["l0.mix.left.q"] == (64, 48) and d["l0.mix.left.q.norm"] == (64,) and d["l0.mix.left.q.b"] == (64,)
    assert d["l0.mix.left.k.norm"] == (32,) and d["l0.mix.left.v.b"] == (16,) and d["l0.mix.left.o.b"] == (48,)
    assert d["l0.mix.right.in"] == (48 + 48 + 16 + 3, 48) and d["l0.mix.right.conv"] == (64, 3)
    assert d["l0.mix.right.conv.b"] == (64,) and d["l0.mix.right.norm"] == (48,) and d["l0.mix.right.o"] == (48, 48)
    assert d["l0.mix.right.A_log"] == d["l0.mix.right.D"] == d["l0.mix.right.dt_bias"] == (3,)
    assert d["l0.mlp.router"] == (5, 48) and d["l0.mlp.e4.down"] == (48, 24) and d["l2.mlp.gate"] == (40, 48)
    assert {"l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "l1.norm1b"} <= set(d) and "l1.norm2" not in d
    assert not any(n.endswith(".out") for n in d)


def test_a_checkpoint_may_hold_the_norms_of_a_missing_feed_forward(tmp_path):
    folder = C.make_model(str(tmp_path), C.A, 3)
    import servelab_b200.weights.source as S
    src = S.FolderSource(folder)

    class More:
        where = "x"

        def names(self):
            return src.names() + ["l1.norm2", "l1.norm2b"]

        def __getattr__(self, n):
            return getattr(src, n)
    CausalLM(config_from_dict(C.A).to_model_spec(), CPU).load(More())


def test_cache_requests_and_flags():
    m = CausalLM(config_from_dict(C.A).to_model_spec(), CPU)
    reqs = m.cache_requests()
    for i, (kv, dim, vdim, window) in enumerate([(2, 16, 8, 5), (1, 8, 24, 33), (2, 24, 16, None)]):
        p = paged_part(reqs[i])
        assert (p.num_kv_heads, p.head_dim, p.value_dim, p.window) == (kv, dim, vdim, window)
    assert [record_floats(r) for r in reqs] == [3 * 8 * 16 + 2 * 64, 4 * 24 * 8 + 1 * (32 + 96), 2 * 16 * 12 + 3 * (24 + 64)]
    for b in m.blocks:
        assert b.graph_safe and b.mixer.padded_steps_safe and part_class(BLOCKS, b.spec).accepts_post_normed


def test_merged_matrices_equal_the_branches():
    """One product in front of both branches, one behind them: columns of a branch begin at a multiple of 8 and
    the columns between are zero; the bias carries the left factor."""
    for cfg in (C.A, C.B):
        spec = config_from_dict(cfg).to_model_spec()
        for i, b in enumerate(spec.layers):
            src = RandomSource(part_class(BLOCKS, b).declare(b, f"l{i}"), 7, dtype=torch.float32)

            class Store:
                def get(self, name):
                    return src.read(name)

                def cat(self, names):
                    return torch.cat([src.read(n) for n in names])
            mix = ParallelMixers(b.mixer, f"l{i}.mix", CPU)
            mix.load(Store())
            lf, rt, pre = b.mixer.left, b.mixer.right, f"l{i}.mix"
            lw, rw = lf.num_heads * lf.value_dim, rt.num_heads * rt.value_dim
            assert mix.right_at % 8 == 0 and mix.row_width % 8 == 0 and mix.right_rows % 8 == 0
            assert torch.equal(mix.w_o[:, :lw], src.read(pre + ".left.o"))
            assert torch.equal(mix.w_o[:, mix.right_at:mix.right_at + rw], src.read(pre + ".right.o"))
            assert float(mix.w_o.abs().sum()) == pytest.approx(
                float(src.read(pre + ".left.o").abs().sum() + src.read(pre + ".right.o").abs().sum()), rel=1e-5)
            assert torch.allclose(mix.o_bias, b.mixer.left_factor * src.read(pre + ".left.o.b"))
            split = 2 * rw + 2 * rt.groups * rt.state_dim
            win = src.read(pre + ".right.in")
            assert torch.equal(mix.w_in[mix.right_rows:mix.right_rows + split], win[:split])
            assert torch.equal(mix.right.w_dt_f32, win[split:])


def test_norm_with_a_factor():
    from servelab_b200.parts.norm import RMSNorm

    class Store:
        def get(self, name):
            return torch.tensor([1.0, -2.0])
    n = RMSNorm(RMSNormSpec(dim=2, factor=0.25, unit_offset=True), "n", CPU)
    n.load(Store())
    assert n.weight.tolist() == [0.5, -0.25]


# ------------------------------------------------------- the oracle's pieces
def test_oracle_slopes_and_sink():
    assert plain.head_slopes(2).tolist() == [2.0 ** -4, 2.0 ** -8]
    # one head, slope 2^-8, no scores: exp(-d/256) over 1 + the sum
    v = torch.tensor([[1.0], [10.0]], dtype=F64).view(2, 1, 1)
    z = torch.zeros(2, 1, 1, dtype=F64)
    o = plain.distance_attention(z, z, v, 1.0, None, None)
    e = math.exp(-1 / 256)
    assert abs(float(o[0]) - 0.5) < 1e-12 and abs(float(o[1]) - (e * 1 + 10) / (2 + e)) < 1e-12
    # the cap acts before the distance is taken off
    q = torch.tensor([0.0, 100.0], dtype=F64).view(2, 1, 1)
    k = torch.ones(2, 1, 1, dtype=F64)
    o = plain.distance_attention(q, k, v, 1.0, 2.0, None)
    s = 2.0 * math.tanh(50.0)
    w0, w1 = math.exp(s - 1 / 256), math.exp(s)
    assert abs(float(o[1]) - (w0 + 10 * w1) / (1 + w0 + w1)) < 1e-12
    assert abs(float(plain.distance_attention(q, k, v, 1.0, 2.0, 1)[1]) - 10 * w1 / (1 + w1)) < 1e-12


def test_oracle_recurrence_and_gated_norm():
    x = torch.tensor([2.0, 3.0], dtype=F64).view(2, 1, 1)
    B = torch.tensor([1.0, 0.5], dtype=F64).view(2, 1, 1)
    Cc = torch.tensor([1.0, 4.0], dtype=F64).view(2, 1, 1)
    dt = torch.tensor([0.5, 2.0], dtype=F64).view(2, 1)
    y = plain.selective_recurrence(x, B, Cc, dt, torch.tensor([math.log(0.25)], dtype=F64), torch.tensor([10.0], dtype=F64))
    s0 = 0.5 * 1.0 * 2.0
    s1 = math.exp(-0.25 * 2.0) * s0 + 2.0 * 0.5 * 3.0
    assert abs(float(y[0]) - (s0 + 20.0)) < 1e-12 and abs(float(y[1]) - (4 * s1 + 30.0)) < 1e-12
    y = torch.tensor([[1.0, 2.0, 3.0, 4.0]], dtype=F64)
    z = torch.tensor([[0.0, 1.0, -1.0, 2.0]], dtype=F64)
    g = [a * b / (1 + math.exp(-b)) for a, b in zip(y[0].tolist(), z[0].tolist())]
    want = [g[0] / math.sqrt((g[0] ** 2 + g[1] ** 2) / 2 + 1e-3), g[1] / math.sqrt((g[0] ** 2 + g[1] ** 2) / 2 + 1e-3),
            g[2] / math.sqrt((g[2] ** 2 + g[3] ** 2) / 2 + 1e-3), g[3] / math.sqrt((g[2] ** 2 + g[3] ** 2) / 2 + 1e-3)]
    got = plain.gated_group_norm(y, z, torch.ones(4, dtype=F64), 2, 1e-3)[0].tolist()
    assert all(abs(a - b) < 1e-12 for a, b in zip(got, want))


def test_oracle_route_and_clamps():
    ids, w = plain.route(torch.tensor([[0.0, 3.0, 3.0, -1.0]], dtype=F64), 2)
    assert ids.tolist() == [[1, 2]] and abs(float(w.sum()) - 2 / (1 + math.exp(-3))) < 1e-12
    y = plain.clamped_unit(torch.tensor([5.0, -5.0], dtype=F64), torch.tensor([-3.0, 3.0], dtype=F64), 2.0)
    assert abs(float(y[0]) - 2 / (1 + math.exp(-3.404)) * -1.0) < 1e-12
    assert abs(float(y[1]) - -5 / (1 + math.exp(1.702 * 5)) * 3.0) < 1e-12
