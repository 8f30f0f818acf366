"""Vufadra on the CPU: config keys and refusals, the spec it turns into, the order its layers run in,
the tensors it declares, what its blocks ask of the cache, pages of chunks, and the oracle's own pieces
on cases worked by hand."""

import copy
import json
import math
import random

import pytest
import torch

import plain_vufadra as plain
import vufadra_cases as C
from servelab_b200.cache import CacheManager
from servelab_b200.cache.manager import PagePool, paged_part, record_floats, state_part
from servelab_b200.cache.storage import CacheStorage, plan_groups
from servelab_b200.config import ConfigError, LayerRun, VufadraConfig, config_from_dict, load_config
from servelab_b200.models.causal_lm import CausalLM, declare_tensors
from servelab_b200.parts import BLOCKS, BuildEnv, part_class

F64 = torch.float64


def test_round_trip_and_registry(tmp_path):
    for cfg, _, _ in C.CASES.values():
        typed = config_from_dict(cfg)
        assert isinstance(typed, VufadraConfig) and typed.to_dict() == cfg
        assert hash(typed) == hash(config_from_dict(copy.deepcopy(cfg)))
    with open(tmp_path / "config.json", "w") as f:
        json.dump(C.A, f)
    assert load_config(str(tmp_path)).to_dict() == C.A


def test_every_size_and_constant_reaches_the_spec():
    spec = config_from_dict(C.A).to_model_spec()
    assert spec.vocab_size == 211 and spec.hidden_size == 48 and not spec.tie_word_embeddings
    assert (spec.bigram.buckets, spec.bigram.mul_prev, spec.bigram.mul_cur) == (101, 31, 7)
    assert spec.loop.times == 3 and spec.logit_scale is None
    assert all(b.kind == "parallel_norm" and b.token_shift and b.mixer_norm.kind == "dynamic_tanh" for b in spec.layers)
    assert [b.mixer.kind for b in spec.layers] == ["parallel_mixers", "gated_recurrence", "delta_rule", "parallel_mixers"]
    assert [b.feed_forward and b.feed_forward.intermediate_size for b in spec.layers] == [40, 24, None, 32]
    par = spec.layers[0].mixer
    assert par.factor == 0.5 and par.eps == 1e-6
    lf, rt = par.left, par.right
    assert (lf.num_heads, lf.num_kv_heads, lf.head_dim, lf.value_dim, lf.scale, lf.chunk, lf.window) == \
        (4, 2, 16, 8, 0.25, 5, None)
    assert lf.weight_fn == "sigmoid" and lf.score_bias and lf.qk_norm and lf.qk_norm_eps == 1e-6 and not lf.sink
    p = lf.position
    assert (p.kind, p.rotary_dim, p.theta, p.yarn_factor, p.yarn_original, p.yarn_fast, p.yarn_slow, p.precise) == \
        ("rotary", 8, 500.0, 4.0, 64.0, 8.0, 1.0, True)
    assert (rt.num_heads, rt.head_dim, rt.value_dim, rt.decay_gate_rank, rt.decay_gate_kind) == (3, 8, 8, 6, "exp_exp")
    assert rt.bonus and rt.token_mix and rt.decay_gate_tanh and not rt.out_norm_per_head and rt.gate_activation == "silu"
    gr = spec.layers[1].mixer
    assert (gr.width, gr.blocks, gr.conv_taps, gr.decay_coef) == (36, 3, 3, 8.0)
    dr = spec.layers[2].mixer
    assert (dr.num_heads, dr.head_dim, dr.value_dim, dr.decay_rank, dr.unit_eps, dr.out_norm_eps) == (3, 8, 8, 5, 1e-6, 1e-6)
    assert abs(dr.decay_coef - math.exp(-0.5)) < 1e-15
    assert spec.layers[3].mixer.left.position.yarn_factor is None
    b = config_from_dict(C.B).to_model_spec()
    assert b.bigram is None and b.loop is None
    assert b.layers[1].mixer.left.position.kind == "none" and b.layers[3].mixer.left.chunk is None


def test_run_order_of_loops():
    run = LayerRun
    assert config_from_dict(C.A).run_order() == (run(0), run(1, None, 0), run(2), run(1, None, 1), run(2),
                                                 run(1, None, 2), run(2), run(3))
    assert config_from_dict(C.B).run_order() == tuple(run(i) for i in range(5))
    assert config_from_dict(C.D).run_order() == (run(0), run(1), run(2, None, 0), run(3))
    assert [i for i, _ in plain.layer_runs(C.C)] == [r.layer for r in config_from_dict(C.C).run_order()]


@pytest.mark.parametrize("change, word", [
    (lambda c: c.update(logit_scale=2.0), "logit_scale"),
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["layers"][1].update(type="mamba"), "mamba"),
    (lambda c: c["layers"][1]["mixer"].update(gate=1), "gate"),
    (lambda c: c["layers"][1]["mixer"].update(blocks=5), "blocks"),
    (lambda c: c["layers"][2]["mixer"].pop("heads"), "heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(first=2), "first"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(low=1), "low"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "moe"),
    (lambda c: c["loop"].update(stop=1), "loop"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c["embedding"].update(norm=1), "norm"),
    (lambda c: c["embedding"]["bigram"].update(buckets=0), "buckets"),
])
def test_refusals_name_the_key(change, word):
    cfg = copy.deepcopy(C.A)
    change(cfg)
    with pytest.raises(ConfigError, match=word):
        config_from_dict(cfg)


def test_declared_tensors():
    decl = {d.name: d.shape for d in declare_tensors(config_from_dict(C.A).to_model_spec())}
    assert decl["bigram"] == (102, 48) and decl["loop.in"] == (48, 96) and decl["loop.step"] == (3, 48)
    assert decl["l0.norm1"] == decl["l0.norm1.b"] == decl["l0.shift"] == (48,) and decl["l0.norm1.alpha"] == ()
    assert decl["l0.mix.left.pb"] == (4,) and decl["l0.mix.left.q.norm"] == (16,) and decl["l0.mix.left.v"] == (16, 48)
    assert decl["l0.mix.right.u"] == (3, 8) and decl["l0.mix.right.mu.w"] == (48,) and decl["l0.mix.right.w2"] == (24, 6)
    assert decl["l0.mix.right.norm"] == (24,) and decl["l0.mix.left.out"] == decl["l0.mix.right.out"] == (48,)
    assert decl["l1.mix.ra"] == (3, 12, 12) and decl["l1.mix.ra.b"] == (3, 12) and decl["l1.mix.conv"] == (36, 3)
    assert decl["l1.mix.y.b"] == decl["l1.mix.lam"] == (36,) and decl["l1.mix.o"] == (48, 36)
    assert decl["l2.mix.a.b"] == decl["l2.mix.w0"] == decl["l2.mix.norm"] == (24,) and decl["l2.mix.w1"] == (5, 48)
    assert "l2.norm2" not in decl and "l2.mlp.up" not in decl and decl["head"] == (211, 48)
    b = {d.name for d in declare_tensors(config_from_dict(C.B).to_model_spec())}
    assert not any(n.startswith(("bigram", "loop")) for n in b)


def test_cache_requests_put_the_records_side_by_side():
    spec = config_from_dict(C.A).to_model_spec()

    def ask(i):
        return part_class(BLOCKS, spec.layers[i]).cache_request(spec.layers[i])
    # the block's own record (the shift), then the mixer's
    assert paged_part(ask(1)) is None and state_part(ask(1)).shape == (48 + 36 + 2 * 36,)
    assert state_part(ask(2)).shape == (48 + 3 * 8 * 8,)
    pages, record = paged_part(ask(0)), state_part(ask(0))
    assert (pages.num_kv_heads, pages.head_dim, pages.value_dim, pages.chunk, pages.window) == (2, 16, 8, 5, None)
    assert record.shape == (48 + 48 + 3 * 8 * 8,) and record_floats(ask(0)) == record.shape[0]
    model = CausalLM(spec, BuildEnv(device="cpu", dtype=torch.float32))
    requests = model.cache_requests()
    assert len(requests) == len(spec.run_order) + 1 and state_part(requests[-1]).shape == (1,)
    storage = CacheStorage(requests, 6, 8, 2, torch.float32, "cpu")
    assert storage.group_chunks == [5, 33] and storage.group_windows == [None, None]
    whole = storage.layer_caches[0]
    part = whole.with_state_slice(48, 48)
    assert part.state.shape == (2, 48) and part.k is whole.k and part.state.stride(0) == record.shape[0]
    assert whole.with_state_slice(48, 0).state is None


def test_pages_of_ended_chunks_go_back():
    pool = PagePool(16, 4, chunk=10)
    pool.open("a")
    pool.grow("a", 26)
    assert pool.trim("a", 9) == [] and pool.num_free() == 9
    assert len(pool.trim("a", 10)) == 2                 # keys 10.. are needed: pages 0 and 1 end before
    assert pool.tables["a"][:3] == [-1, -1, 2]
    assert pool.trim("a", 19) == [] and len(pool.trim("a", 25)) == 3      # keys 20.. are needed
    assert pool.peak_pages(1000, 7) == 6 and pool.peak_pages(8, 7) == 2
    pool.close("a")
    assert pool.num_free() == 16
    with pytest.raises(ValueError):
        PagePool(4, 4, window=3, chunk=5)
    # a reader at any later position finds every page it needs
    rng = random.Random(3)
    for _ in range(50):
        chunk, page, cm = rng.randint(1, 40), rng.choice([2, 4, 8]), None
        cm = CacheManager([None, None], 200, page, 3, group_chunks=[chunk, None])
        held = {}
        for _ in range(60):
            rid = f"r{rng.randint(0, 3)}"
            if rid not in held and not cm.open(rid):
                continue
            held.setdefault(rid, 0)
            n = rng.randint(1, 15)
            if not cm.ensure(rid, held[rid] + n):
                continue
            start = held[rid]
            table = cm.block_table(rid, 0)
            for q in range(start, start + n):
                for k in range(q - q % chunk, q + 1):
                    assert table[k // page] >= 0
            held[rid] += n
            cm.trim(rid, held[rid])
            cm.check_invariants()
            if rng.random() < 0.15:
                cm.release(rid)
                held.pop(rid)
    groups, _ = plan_groups(CausalLM(config_from_dict(C.D).to_model_spec(),
                                     BuildEnv(device="cpu", dtype=torch.float32)).cache_requests())
    assert [g.request.chunk for g in groups] == [1000, 40]


# ------------------------------------------------------ the oracle by hand
def test_plain_bigram_rows_and_shift():
    assert plain.bigram_rows([4, 9, 4], 10, 3, 7) == [10, (4 * 3 + 9 * 7) % 10, (9 * 3 + 4 * 7) % 10]
    h = torch.tensor([[2.0], [6.0], [1.0]], dtype=F64)
    assert plain.token_shift(h, torch.tensor([0.25], dtype=F64))[:, 0].tolist() == [1.5, 5.0, 2.25]


def test_plain_attention_sees_its_chunk_only():
    m = plain.visible_in_chunk(7, 3)
    assert m[4].tolist() == [False, False, False, True, True, False, False] and m[6].sum() == 1
    q = torch.zeros(5, 1, 2, dtype=F64)
    v = torch.arange(1.0, 6.0, dtype=F64).view(5, 1, 1)
    o = plain.sigmoid_attention(q, q, v, 1.0, torch.tensor([0.0]), 2)[:, 0, 0]
    assert o.tolist() == [0.5, 1.5, 1.5, 3.5, 2.5]


def test_plain_delta_rule_replaces_a_key():
    k = torch.tensor([[[2.0, 0.0]], [[0.0, 1.0]], [[2.0, 0.0]]], dtype=F64)
    v = torch.tensor([[[1.0]], [[5.0]], [[3.0]]], dtype=F64)
    one, r = torch.ones(3, 1, 2, dtype=F64), torch.tensor([[[1.0, 1.0]]] * 3, dtype=F64)
    assert torch.allclose(plain.delta_rule(r, k, v, one, one)[:, 0, 0], torch.tensor([2.0, 7.0, 11.0], dtype=F64), atol=1e-5)
    assert torch.allclose(plain.delta_rule(r, k, v, one, 0 * one)[:, 0, 0], torch.tensor([2.0, 7.0, 13.0], dtype=F64))


def test_plain_bonus_and_gated_unit():
    one = torch.ones(2, 1, 1, dtype=F64)
    o = plain.bonus_recurrence(one, one, 3 * one, 0.5 * one, torch.tensor([[10.0]], dtype=F64))
    assert o[:, 0, 0].tolist() == [30.0, 33.0]
    r = torch.tensor([[0.0], [1e9]], dtype=F64)
    S = plain.gated_unit(torch.full((2, 1), 4.0, dtype=F64), r, torch.ones(2, 1, dtype=F64), torch.tensor([0.0], dtype=F64))
    assert S[:, 0].tolist() == [0.0, 4.0]               # a = 1 lets nothing in, a = 0 forgets everything


def test_plain_ramp_and_block_diagonal():
    f, mag = plain.yarn_frequencies(8, 100.0, {"factor": 4.0, "original": 16, "fast": 1e6, "slow": 1e-6})
    assert abs(mag - (0.1 * math.log(4.0) + 1.0)) < 1e-12
    plainf, _ = plain.yarn_frequencies(8, 100.0, None)
    assert f[0] == plainf[0] and f[-1] < plainf[-1]
    w = torch.stack([torch.eye(2, dtype=F64), 2 * torch.eye(2, dtype=F64)])
    out = plain.block_linear(torch.ones(1, 4, dtype=F64), w, torch.zeros(2, 2, dtype=F64))
    assert out.tolist() == [[1.0, 1.0, 2.0, 2.0]]
