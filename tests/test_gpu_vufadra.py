"""Vufadra on the GPU against the plain implementation (``plain_vufadra``): every new mechanism alone,
then whole models replayed whole, token by token, in portions down to two tokens and in mixed batches
with pages and slots used again, in float32 and bfloat16, and greedy generation through the engine."""

import numpy as np
import pytest
import torch

import helpers as H
import plain_vufadra as plain
import vufadra_cases as C

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64
BOTH = [torch.float32, torch.bfloat16]


def _ctx(entries, groups=1):
    from servelab_b200.engine.batch import StepContext
    return StepContext.pack(entries, groups, DEV)


def _entry(tokens, start, table=(), slot=0):
    from servelab_b200.engine.batch import BatchEntry
    ids = tokens if isinstance(tokens, list) else [0] * tokens
    return BatchEntry(tokens=ids, start=start, want=(), block_tables=[list(table)], state_slot=slot)


def _padded_ctx(entries, tokens, seqs):
    from servelab_b200.engine.batch import StepContext
    return StepContext.pack(entries, 0, DEV, pad=(tokens, seqs, 0))


def _close(got, want, tol, what=""):
    scale = max(1.0, float(want.abs().max()))
    err = float((got.double().cpu() - want).abs().max()) / scale
    assert err < tol, (what, err)


# steps of one request of n tokens in slot 0 and one of m in slot 2: (slot, first row, rows) a piece
def _schedules(n, m):
    whole = [[(0, 0, n), (2, n, m)]]
    portions = [[(0, 0, 2)], [(2, n, 1), (0, 2, n - 7)], [(0, n - 5, 2)], [(0, n - 3, 1), (2, n + 1, m - 1)], [(0, n - 2, 2)]]
    single = [[(0, i, 1)] + ([(2, n + i, 1)] if i < m else []) for i in range(n)]
    return {"whole": whole, "portions": portions, "single": single}


def _run(schedule, state, body, n):
    """``body(rows, ctx)`` runs a step on the given rows; slots are zeroed where a request begins."""
    outs = {}
    for step in schedule:
        for slot, a, k in step:
            if a in (0, n):
                state[slot].zero_()
        rows = torch.cat([torch.arange(a, a + k) for _, a, k in step])
        ctx = _ctx([_entry(k, a - (0 if a < n else n), (), slot) for slot, a, k in step], 0)
        o = body(rows, ctx)
        for i, r in enumerate(rows.tolist()):
            outs[r] = o[..., i, :]
    return torch.stack([outs[r] for r in sorted(outs)], dim=-2)


# --------------------------------------------------------------- embedding
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("muls", [(101, 31, 7), (1, 5, 3), (7, 10 ** 9 + 7, 998244353)])
def test_bigram_embedding_follows_the_previous_token(dtype, muls):
    """Whole, in portions and token by token, two requests a step, a slot used again, and padding that
    must leave the records alone; products beyond 32 bits."""
    from servelab_b200.ops import kernels as K
    buckets, mp, mc = muls
    g = torch.Generator().manual_seed(1)
    V, w = 90000, 36
    table = torch.randn(V, w, generator=g).to(dtype)
    pairs = torch.randn(buckets + 1, w, generator=g).to(dtype)
    ids = torch.randint(0, V, (29,), generator=g).tolist()
    n = 20
    want = torch.cat([table[torch.tensor(s)].double() + pairs[torch.tensor(plain.bigram_rows(s, buckets, mp, mc))].double()
                      for s in (ids[:n], ids[n:])])
    tab, prs = table.to(DEV), pairs.to(DEV)
    state = torch.zeros(3, 1, device=DEV)
    for name, schedule in _schedules(n, 9).items():
        def body(rows, ctx):
            ctx.token_ids.copy_(torch.tensor([ids[r] for r in rows.tolist()], dtype=torch.int32))
            out = torch.empty(len(rows), w, device=DEV)
            both = torch.zeros(len(rows), 2 * w, dtype=dtype, device=DEV)
            K.embed_bigram(ctx, tab, prs, buckets, mp, mc, state, out, both[:, w:])
            assert torch.equal(both[:, w:], out.to(dtype)) and float(both[:, :w].abs().max()) == 0
            return out
        got = _run(schedule, state, body, n)
        _close(got, want, 1e-6, name)
        assert state.view(torch.int32)[:, 0].tolist() == [ids[n - 1] + 1, 0, ids[-1] + 1]
    ctx = _padded_ctx([_entry([5, 6], 0, (), 1)], 16, 2)
    out = torch.empty(16, w, device=DEV)
    K.embed_bigram(ctx, tab, prs, buckets, mp, mc, state, out)
    assert state.view(torch.int32)[:, 0].tolist() == [ids[n - 1] + 1, 7, ids[-1] + 1]


# ------------------------------------------------- norms, shift, side by side
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("w", [48, 50, 1028])
@pytest.mark.parametrize("many", [False, True])
def test_two_norms_side_by_side_with_a_token_shift(dtype, w, many):
    """Pending updates of both types and a row for every token are added, both norms formed, the first
    mixed with the previous token's; the record holds the last token's norm before the mix."""
    from servelab_b200.ops import kernels as K
    g = torch.Generator().manual_seed(w)
    n, m = (700, 300) if many else (20, 9)
    T = n + m
    resid = torch.randn(T, w, generator=g)
    d1 = torch.randn(T, w, generator=g).to(dtype)
    d2 = torch.randn(T, w, generator=g)
    row = torch.randn(w, generator=g)
    n1 = (torch.tensor([0.7]), torch.randn(w, generator=g), torch.randn(w, generator=g))
    n2 = (torch.tensor([1.3]), torch.randn(w, generator=g), torch.randn(w, generator=g))
    shift = torch.randn(w, generator=g)
    x = resid.double() + d1.double() + d2.double() + row.double()
    h = plain.dynamic_tanh(x, *(t.double() for t in n1))
    want1 = torch.cat([plain.token_shift(h[:n], shift.double()), plain.token_shift(h[n:], shift.double())])
    want2 = plain.dynamic_tanh(x, *(t.double() for t in n2))
    dev = [t.to(DEV) for t in (resid, d1, d2, row, shift)]
    p1, p2 = tuple(t.to(DEV) for t in n1), tuple(t.to(DEV) for t in n2)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    ws = -(-w // 4) * 4
    schedules = _schedules(n, m)
    if many:
        schedules = {"whole": schedules["whole"]}
    for name, schedule in schedules.items():
        big = torch.full((3, ws + 8), 3.0, device=DEV)
        prev = big[:, 4:4 + ws]

        def body(rows, ctx):
            r, a, b = dev[0][rows].contiguous(), dev[1][rows].contiguous(), dev[2][rows].contiguous()
            o1 = torch.empty(len(rows), w, dtype=dtype, device=DEV)
            o2, xo = torch.empty_like(o1), torch.empty_like(r)
            K.dyt_parallel(ctx, r, (a, b), dev[3], p1, o1, p2, o2, xo, dev[4], prev)
            return torch.cat([o1.float(), o2.float(), xo], dim=1)
        got = _run(schedule, prev, body, n)
        _close(got[:, :w], want1, tol, name)
        _close(got[:, w:2 * w], want2, tol, name)
        _close(got[:, 2 * w:], x, 1e-5, name)
        _close(prev[[0, 2], :w], h[[n - 1, T - 1]], 1e-5, name)
        assert float(big[:, :4].min()) == 3.0 and float(big[:, 4 + ws:].min()) == 3.0
    keep = prev.clone()
    ctx = _padded_ctx([_entry(2, 0, (), 1)], 16, 2)
    o1 = torch.empty(16, w, dtype=dtype, device=DEV)
    K.dyt_parallel(ctx, dev[0][:16].contiguous(), (), None, p1, o1, shift=dev[4], prev=prev)
    assert torch.equal(prev[[0, 2]], keep[[0, 2]]) and not torch.equal(prev[1], keep[1])
    # the norm of selected rows, and the stream as an operand
    rows = torch.tensor([3, T - 1, 0], dtype=torch.int32, device=DEV)
    o = torch.empty(3, w, dtype=dtype, device=DEV)
    K.dyt_parallel(ctx, dev[0], (dev[1], dev[2]), dev[3], p2, o, row_map=rows)
    _close(o, want2[rows.long().cpu()], tol)
    both = torch.zeros(T, 2 * w, dtype=dtype, device=DEV)
    K.stream_rows(dev[0], (dev[2],), dev[3], both[:, :w])
    _close(both[:, :w], resid.double() + d2.double() + row.double(), tol)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("w", [48, 50, 1028])
def test_mixes_with_the_previous_token(dtype, w):
    from servelab_b200.ops import kernels as K
    g = torch.Generator().manual_seed(w)
    n, m = 20, 9
    x = torch.randn(n + m, w, generator=g).to(dtype)
    mu = torch.randn(5, w, generator=g)
    want = torch.stack([torch.cat([plain.token_shift(x[:n].double(), v.double()),
                                   plain.token_shift(x[n:].double(), v.double())]) for v in mu])
    xd, md = x.to(DEV), mu.to(DEV)
    prev = torch.full((3, -(-w // 4) * 4), 3.0, device=DEV)
    for name, schedule in _schedules(n, m).items():
        def body(rows, ctx):
            out = torch.empty(5, len(rows), w, dtype=dtype, device=DEV)
            K.token_mix(ctx, xd[rows].contiguous(), md, prev, out)
            return out
        _close(_run(schedule, prev, body, n), want, 1e-5 if dtype == torch.float32 else 1e-2, name)
    keep = prev.clone()
    out = torch.empty(5, 16, w, dtype=dtype, device=DEV)
    K.token_mix(_padded_ctx([_entry(2, 0, (), 1)], 16, 2), xd[:16].contiguous(), md, prev, out)
    assert torch.equal(prev[[0, 2]], keep[[0, 2]]) and not torch.equal(prev[1], keep[1])


def test_interpolated_frequencies_of_a_half_split_rotation():
    from servelab_b200.config.specs import RotarySpec
    from servelab_b200.parts import BuildEnv
    from servelab_b200.parts.position import RotaryEmbedding
    env = BuildEnv(device="cpu", dtype=torch.float32)
    for dims, base, sc in ((16, 2e6, (4.0, 512, 32.0, 1.0)), (32, 1e4, (8.0, 32, 4.0, 0.5)), (8, 500.0, (4.0, 64, 8.0, 1.0)),
                           (64, 5e5, (1.0, 4096, 32.0, 1.0)), (2, 1e4, (2.0, 64, 1.0, 1.0))):
        spec = RotarySpec(head_dim=dims, rotary_dim=dims, theta=base, yarn_factor=sc[0], yarn_original=sc[1],
                          yarn_fast=sc[2], yarn_slow=sc[3], precise=True)
        part = RotaryEmbedding(spec, "x", env)
        want, mag = plain.yarn_frequencies(dims, base, dict(zip(("factor", "original", "fast", "slow"), sc)))
        f, _ = part.rotary_table()
        assert (f.double() - want).abs().max() <= 1e-7 * want.abs().max() and abs(part.magnitude - mag) < 1e-12


# --------------------------------------- attention: chunks and sigmoid weights
def _attention_case(seed, Hq, G, Dk, Dv, chunk, ctxs, qlens, ps, dtype, spike, bias):
    """Requests with contexts ``ctxs`` whose last ``qlens`` tokens are this step's queries; keys and
    values in pages in a shuffled order (unwritten slots hold a huge number).  ``spike`` = "in": the
    first key of every chunk gets a score far above the others and a value of its own (it counts for
    the whole chunk); "out": the last key of every chunk does (for the next chunk it must not)."""
    g = torch.Generator().manual_seed(seed)
    n_pages = sum(-(-c // ps) for c in ctxs) + 3
    order = torch.randperm(n_pages, generator=g).tolist()
    kc = torch.full((n_pages, G, ps, Dk), 1e30, dtype=dtype)
    vc = torch.full((n_pages, G, ps, Dv), 1e30, dtype=dtype)
    qs, wants, entries = [], [], []
    for c, n in zip(ctxs, qlens):
        k = torch.randn(c, G, Dk, generator=g) * 0.5
        v = torch.randn(c, G, Dv, generator=g)
        q = torch.randn(n, Hq, Dk, generator=g) * 0.5
        if spike is not None:
            size = chunk or c
            q[..., 0] = 2.0                            # what the marked keys answer to ...
            k[..., 0] = -2.0                           # ... and the others do not
            at = list(range(0 if spike == "in" else size - 1, c, size))
            k[at, :, 0] = 6.0
            v[at] = 7.0
        k, v, q = k.to(dtype), v.to(dtype), q.to(dtype)
        table = [order.pop() for _ in range(-(-c // ps))]
        for p in range(c):
            kc[table[p // ps], :, p % ps] = k[p]
            vc[table[p // ps], :, p % ps] = v[p]
        if chunk:                                      # pages of ended chunks have gone back
            first = (c - n) - (c - n) % chunk
            for lp in range(first // ps):
                kc[table[lp]], vc[table[lp]] = 1e30, 1e30
                table[lp] = -1
        qfull = torch.zeros(c, Hq, Dk, dtype=F64)
        qfull[c - n:] = q.double()
        o = plain.sigmoid_attention(qfull, k.double(), v.double(), 0.2, bias, chunk)
        wants.append(o[c - n:].reshape(n, Hq * Dv))
        qs.append(q.reshape(n, Hq * Dk))
        entries.append(_entry(n, c - n, table))
    return {"q": torch.cat(qs).to(DEV), "kc": kc.to(DEV), "vc": vc.to(DEV), "want": torch.cat(wants), "entries": entries}


SHAPES = [(4, 2, 80, 48, 0), (5, 1, 112, 96, 40), (3, 3, 10, 6, 9), (8, 2, 64, 64, 90), (6, 1, 128, 128, 1),
          (4, 2, 32, 32, 33), (2, 1, 160, 128, 300), (16, 2, 64, 128, 70), (1, 1, 64, 64, 64), (34, 2, 16, 16, 128)]


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("spike", ["in", "out", None])
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("decode", [False, True])
def test_attention_in_chunks_with_sigmoid_weights(dtype, spike, shape, decode):
    """Portions and single tokens at page, tile and chunk edges, the first token of a chunk, a portion
    over several chunks, heads whose bias opens or closes every key."""
    from servelab_b200.ops import attention as A
    from servelab_b200.ops import kernels as K
    Hq, G, Dk, Dv, chunk = shape
    ps = 8
    c = chunk or 64
    ctxs = [1, 2, 300, 301, 64, 65, 333, c, c + 1, 2 * c, 2 * c + 1]
    qlens = [1] * len(ctxs) if decode else [1, 2, 200, 37, 64, 3, 33, c, 2, c + 1, 1]
    bias = torch.linspace(-3.0, 2.0, Hq)
    case = _attention_case(7, Hq, G, Dk, Dv, chunk, ctxs, qlens, ps, dtype, spike, bias)
    ctx = _ctx(case["entries"])

    def run():
        out = torch.empty(case["q"].shape[0], Hq * Dv, dtype=dtype, device=DEV)
        A.kv_attention(ctx, case["q"], case["kc"], case["vc"], Dv, out, ctx.block_tables[0], Hq, G, Dk, Dv,
                       ps, 0.2, 0, None, chunk=chunk, sigmoid_bias=bias.to(DEV))
        return out
    tol = 1e-5 if dtype == torch.float32 else 1.5e-2
    _close(run(), case["want"], tol)
    if dtype == torch.bfloat16:
        A.force_generic = True                         # the plain kernel is the twin of the tensor-core ones ...
        try:
            _close(run(), case["want"], tol, "plain")
        finally:
            A.force_generic = False
        A.use_kv_tc_capped = False                     # ... and mma.sync the twin of tcgen05
        try:
            _close(run(), case["want"], tol, "mma")
        finally:
            A.use_kv_tc_capped = True
        if Dk % 64 == 0 and Dv % 64 == 0:
            assert K.attention_kv_tc_status(Dk, Dv) == 0 and K.attention_kv_mma_status(Dk, Dv) == 0


def test_attention_single_tokens_with_key_splits_and_sigmoid_weights():
    """Few requests with long contexts: the keys are split over blocks, whose results add up."""
    from servelab_b200.ops import attention as A
    for chunk, ctxs in ((0, [1500, 900, 1]), (1100, [1100, 2201, 900])):
        Hq, G, Dk, Dv, ps = 8, 2, 64, 48, 16
        bias = torch.linspace(-4.0, 1.0, Hq)
        case = _attention_case(5, Hq, G, Dk, Dv, chunk, ctxs, [1, 1, 1], ps, torch.bfloat16, "in", bias)
        ctx = _ctx(case["entries"])
        out = torch.empty(3, Hq * Dv, dtype=torch.bfloat16, device=DEV)
        A.kv_attention(ctx, case["q"], case["kc"], case["vc"], Dv, out, ctx.block_tables[0], Hq, G, Dk, Dv, ps, 0.2, 0,
                       None, chunk=chunk, sigmoid_bias=bias.to(DEV))
        _close(out, case["want"], 1.5e-2, chunk)


# ------------------------------------------------------------- recurrences
def _lens(n, m):
    return [(0, n), (n, n + m)]


DELTA_SHAPES = [(3, 8, 8), (2, 40, 64), (1, 64, 64), (2, 128, 128), (1, 136, 33), (2, 14, 10), (1, 256, 300), (1, 130, 256)]


def _delta_case(seed, Hh, D, Dv, T, dtype, slow=False):
    g = torch.Generator().manual_seed(seed)
    proj = torch.randn(T, 3 * Hh * D + 2 * Hh * Dv + 5, generator=g).to(dtype)
    z = torch.randn(T, Hh * D, generator=g) * 2 - (9.0 if slow else 0.0)
    return proj, z, torch.randn(Hh * D, generator=g) - (2.0 if slow else 0.0), torch.randn(Hh * Dv, generator=g)


def _delta_want(case, Hh, D, Dv, lens, coef, eps):
    proj, z, ab, nw = (t.double() for t in case)
    outs = []
    for a0, a1 in lens:
        p, n = proj[a0:a1], a1 - a0
        qs, vs = Hh * D, Hh * Dv
        r, k = p[:, :qs].view(n, Hh, D), p[:, qs:2 * qs].view(n, Hh, D)
        v, gate = p[:, 2 * qs:2 * qs + vs].view(n, Hh, Dv), p[:, 2 * qs + vs:2 * qs + 2 * vs]
        a = torch.sigmoid(p[:, 2 * qs + 2 * vs:3 * qs + 2 * vs] + ab).view(n, Hh, D)
        w = torch.exp(-coef * torch.sigmoid(z[a0:a1])).view(n, Hh, D)
        o = plain.rms_norm(plain.delta_rule(r, k, v, w, a), None, eps).reshape(n, vs)
        outs.append(o * nw * torch.sigmoid(gate))
    return torch.cat(outs)


def _run_delta(K, case, Hh, D, Dv, rows, ctx, state, coef, eps):
    proj, z, ab, nw = case
    out = torch.empty(len(rows), Hh * Dv, dtype=proj.dtype, device=DEV)
    qs, vs = Hh * D, Hh * Dv
    K.delta_rule(ctx, proj[rows].contiguous(), state, out, r_off=0, k_off=qs, v_off=2 * qs, g_off=2 * qs + vs,
                 a_off=2 * qs + 2 * vs, num_heads=Hh, head_dim=D, value_dim=Dv, a_bias=ab, gate_z=z[rows].contiguous(),
                 decay_coef=coef, unit_eps=1e-6, norm_w=nw, norm_eps=eps)
    return out


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("shape", DELTA_SHAPES)
def test_delta_rule_whole_in_portions_and_token_by_token(dtype, shape, monkeypatch):
    """The token-by-token kernel: its results do not depend on the cut, bit for bit; the record may be a
    slice of a larger one."""
    from servelab_b200.ops import kernels as K
    monkeypatch.setattr(K, "delta_rule_chunked", False)
    Hh, D, Dv = shape
    n, m = 41, 7
    host = _delta_case(3, Hh, D, Dv, n + m, dtype)
    want = _delta_want(host, Hh, D, Dv, _lens(n, m), 0.6, 1e-5)
    case = tuple(t.to(DEV) for t in host)
    rec = Hh * D * Dv
    results = []
    for name, schedule in _schedules(n, m).items():
        big = torch.full((3, rec + 8), 3.0, device=DEV)
        state = big[:, 4:4 + rec]
        got = _run(schedule, state, lambda rows, ctx: _run_delta(K, case, Hh, D, Dv, rows, ctx, state, 0.6, 1e-5), n)
        _close(got, want, 5e-5 if dtype == torch.float32 else 1e-2, name)
        assert float(big[:, :4].min()) == 3.0 and float(big[:, 4 + rec:].min()) == 3.0
        results.append((got, state[[0, 2]].clone()))
    for got, st in results[1:]:
        assert torch.equal(got, results[0][0]) and torch.equal(st, results[0][1])


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("shape", DELTA_SHAPES)
@pytest.mark.parametrize("slow", [False, True])
def test_delta_rule_in_chunks(dtype, shape, slow, monkeypatch):
    """The chunked kernels: requests shorter than a chunk, a chunk exactly, a chunk and one token,
    several chunks, cuts inside chunks, the state they leave against the token-by-token kernel's."""
    from servelab_b200.ops import kernels as K
    monkeypatch.setattr(K, "force_delta_chunks", True)
    monkeypatch.setattr(K, "delta_rule_chunk_min_tokens", 1)
    Hh, D, Dv = shape
    lens = [5, 32, 33, 131]
    starts = [0, 5, 37, 70]
    T = sum(lens)
    host = _delta_case(11, Hh, D, Dv, T, dtype, slow)
    want = _delta_want(host, Hh, D, Dv, [(a, a + k) for a, k in zip(starts, lens)], 0.6065, 1e-5)
    case = tuple(t.to(DEV) for t in host)
    rec = Hh * D * Dv
    big = torch.full((4, rec + 8), 3.0, device=DEV)
    state = big[:, 4:4 + rec]
    state.zero_()

    def step(pieces):
        rows = torch.cat([torch.arange(a, a + k) for _, a, k in pieces])
        ctx = _ctx([_entry(k, 0, (), slot) for slot, a, k in pieces], 0)
        return rows, _run_delta(K, case, Hh, D, Dv, rows, ctx, state, 0.6065, 1e-5)
    tol = 1e-4 if dtype == torch.float32 else 1e-2
    _, got = step([(s, a, k) for s, (a, k) in enumerate(zip(starts, lens))])
    _close(got, want, tol)
    assert float(big[:, :4].min()) == 3.0 and float(big[:, 4 + rec:].min()) == 3.0
    final = state.clone()
    state.zero_()
    a = 70
    for k in (45, 16, 53, 2, 15):
        rows, got = step([(3, a, k)])
        _close(got, want[rows], tol, a)
        a += k
    _close(state[3], final[3].double().cpu(), 1e-4, "cut")
    state.zero_()
    monkeypatch.setattr(K, "force_delta_chunks", False)
    monkeypatch.setattr(K, "delta_rule_chunked", False)
    step([(3, 70, 131)])
    _close(state[3], final[3].double().cpu(), 1e-4, "token by token")


def test_delta_rule_keeps_replaces_and_forgets():
    """One key 900 tokens back, asked for by the last query.  Without decay and removal it still answers; a
    later token with the same key and full removal replaces its value; decay forgets it.  Chunked,
    token by token and both."""
    from servelab_b200.ops import kernels as K
    D, Dv, T = 16, 8, 901
    Hh = 3
    qs, vs = Hh * D, Hh * Dv
    proj = torch.zeros(T, 3 * qs + 2 * vs)
    for h in range(Hh):
        proj[0, qs + h * D] = 1.0                                  # the key e_0 ...
        proj[0, 2 * qs + h * Dv:2 * qs + (h + 1) * Dv] = torch.arange(1.0, 9.0)      # ... and its value
        proj[T - 1, h * D] = 1.0                                   # the query
    proj[:, 2 * qs + 2 * vs:] = -30.0                              # removal rates 0 ...
    proj[450, qs + D] = 1.0                                        # head 1: the same key again ...
    proj[450, 2 * qs + Dv:2 * qs + 2 * Dv] = torch.arange(8.0, 0.0, -1.0)
    proj[450, 2 * qs + 2 * vs + D:2 * qs + 2 * vs + 2 * D] = 30.0  # ... with full removal
    z = torch.full((T, qs), -30.0)                                 # no decay
    z[:, 2 * D:] = -3.0                                            # head 2: exp(-0.6 sigmoid(-3)) a step
    case = tuple(t.to(DEV) for t in (proj.to(torch.bfloat16), z, torch.zeros(qs), torch.ones(vs)))
    one = torch.arange(1.0, 9.0, dtype=F64)
    for cuts in ([901], [1] * 901, [400, 1, 30, 70, 400]):
        state = torch.zeros(1, Hh * D * Dv, device=DEV)
        a = 0
        for k in cuts:
            rows = torch.arange(a, a + k)
            out = _run_delta(K, case, Hh, D, Dv, rows, _ctx([_entry(k, a)], 0), state, 0.6, 1e-12)
            a += k
        last = out[-1].double().cpu().view(Hh, Dv)
        norm = one / (one * one).mean().sqrt() * 0.5               # (the gate is sigmoid(0))
        assert (last[0] - norm).abs().max() < 2e-2 and (last[1] - norm.flip(0)).abs().max() < 2e-2
        assert state.view(Hh, D, Dv)[2].abs().max() < 1e-8


BONUS_SHAPES = [(3, 8), (2, 64), (1, 24), (2, 136), (1, 10)]


def _bonus_case(seed, Hh, D, T, dtype, shift):
    g = torch.Generator().manual_seed(seed)
    proj = (torch.randn(T, 3 * Hh * D + 5, generator=g) * 0.5).to(dtype)
    return proj, torch.randn(T, Hh * D, generator=g) * 2 + shift, torch.randn(Hh * D, generator=g), torch.randn(Hh * D, generator=g)


def _bonus_want(case, Hh, D, lens):
    proj, z, bias, u = (t.double() for t in case)
    outs = []
    for a0, a1 in lens:
        n = a1 - a0
        r, k, v = (proj[a0:a1, i * Hh * D:(i + 1) * Hh * D].view(n, Hh, D) for i in range(3))
        w = torch.exp(-torch.exp(z[a0:a1] + bias)).view(n, Hh, D)
        outs.append(plain.bonus_recurrence(r, k, v, w, u.view(Hh, D)).reshape(n, Hh * D))
    return torch.cat(outs)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("shape", BONUS_SHAPES)
@pytest.mark.parametrize("shift", [-4.0, 0.0, 4.0])
def test_recurrence_with_a_bonus_and_double_exponential_decays(dtype, shape, shift, monkeypatch):
    """Token by token (bit for bit independent of the cut) and in chunks, from slow decays to such that a
    channel is gone after a token (also logits whose exponential leaves float32)."""
    from servelab_b200.ops import kernels as K
    Hh, D = shape
    n, m = 75, 7
    host = list(_bonus_case(21, Hh, D, n + m, dtype, shift))
    if shift > 0:
        host[1][3] = 200.0
    want = _bonus_want(host, Hh, D, _lens(n, m))
    proj, z, bias, u = (t.to(DEV) for t in host)
    rec = Hh * D * D

    def body(state):
        def run(rows, ctx):
            o = torch.empty(len(rows), Hh * D, dtype=torch.float32, device=DEV)
            K.decay_attention(proj[rows].contiguous(), ctx, state, None, o, q_off=0, k_off=Hh * D, v_off=2 * Hh * D,
                              num_heads=Hh, head_dim=D, value_dim=D, gate_z=z[rows].contiguous(), gate_bias=bias,
                              gate_kind="exp_exp", bonus=u)
            return o
        return run
    results = []
    for chunks in (False, True):
        monkeypatch.setattr(K, "decay_gated_chunked", chunks)
        monkeypatch.setattr(K, "force_gated_chunks", chunks)
        monkeypatch.setattr(K, "decay_attention_chunk_min_tokens", 1)
        for name, schedule in _schedules(n, m).items():
            big = torch.full((3, rec + 8), 3.0, device=DEV)
            state = big[:, 4:4 + rec]
            got = _run(schedule, state, body(state), n)
            _close(got, want, 3e-5, (name, chunks))
            assert float(big[:, :4].min()) == 3.0 and float(big[:, 4 + rec:].min()) == 3.0
            if not chunks:
                results.append((got, state[[0, 2]].clone()))
            else:
                _close(state[[0, 2]], results[0][1].double().cpu(), 3e-5)
    for got, st in results[1:]:
        assert torch.equal(got, results[0][0]) and torch.equal(st, results[0][1])


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("shape", [(36, 3, 3), (30, 5, 1), (128, 1, 5), (96, 6, 2), (1040, 2, 4), (17, 1, 2)])
@pytest.mark.parametrize("segments", [False, True])
def test_gated_recurrence_with_its_convolution(dtype, shape, segments, monkeypatch):
    """Convolution with its biases (whose zeros before the start stay zeros), block-diagonal gates and the
    recurrence: whole, in portions, token by token, decays near 1 and fast ones; with `segments` the
    kernel that takes longer portions 256 tokens at a time."""
    from servelab_b200.ops import kernels as K
    from servelab_b200.config.specs import GatedRecurrenceSpec
    from servelab_b200.parts import BuildEnv, LayerCache
    from servelab_b200.parts.gated_recurrence import GatedRecurrence
    width, blocks, taps = shape
    hidden, n, m = 40, 530 if segments else 150, 9
    monkeypatch.setattr(K, "force_gated_recurrence_segments", segments)
    g = torch.Generator().manual_seed(width)
    spec = GatedRecurrenceSpec(hidden_size=hidden, width=width, blocks=blocks, conv_taps=taps)
    W = {}
    for d in GatedRecurrence.declare(spec, "m"):
        std = {"m.lam": 3.0, "m.conv": 0.6}.get(d.name, 0.5 if d.name.endswith(".b") else 0.3)
        W[d.name] = (torch.randn(d.shape, generator=g) * std).to(torch.bfloat16)

    class Store:
        def get(self, name):
            dt = dtype if name in ("m.y", "m.x", "m.ra", "m.ri", "m.o") else torch.float32
            return W[name].to(DEV, dt).contiguous()

        def cat(self, names):
            return torch.cat([self.get(x) for x in names])
    mixer = GatedRecurrence(spec, "m", BuildEnv(device=DEV, dtype=dtype))
    mixer.load(Store())
    mixer.out_dtype = torch.float32
    x = torch.randn(n + m, hidden, generator=g).to(dtype)
    want = torch.cat([plain.rglru_mixer(x[:n].double(), W, "m"), plain.rglru_mixer(x[n:].double(), W, "m")])
    (floats,) = GatedRecurrence.cache_request(spec).shape
    xd = x.to(DEV)
    results = []
    for name, schedule in _schedules(n, m).items():
        state = torch.full((3, floats), 3.0, device=DEV)
        got = _run(schedule, state, lambda rows, ctx: mixer.forward(ctx, xd[rows].contiguous(), LayerCache(state=state), True), n)
        _close(got, want, 1e-5 if dtype == torch.float32 else 2e-2, name)
        assert float(state[1].min()) == 3.0
        results.append(got)
    if dtype == torch.float32 and not segments:
        assert torch.equal(results[0], results[1]) and torch.equal(results[0], results[2])
    keep = state.clone()
    mixer.forward(_padded_ctx([_entry(2, 0, (), 1)], 16, 2), xd[:16].contiguous(), LayerCache(state=state), True)
    assert torch.equal(state[[0, 2]], keep[[0, 2]]) and not torch.equal(state[1], keep[1])


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("shape", [(1, 64, 8, 0), (9, 40, 24, 0), (70, 130, 64, 8), (65, 33, 13, 3), (600, 200, 72, 16),
                                   (520, 131, 7, 1)])
def test_second_product_of_a_bottleneck(dtype, shape):
    """tanh kept to more than the operands' 8 bits; columns of a larger projection; sizes of no tile."""
    from servelab_b200.ops import kernels as K
    M, N, R, off = shape
    g = torch.Generator().manual_seed(M)
    proj = torch.randn(M, R + 2 * off + 8, generator=g).to(dtype)
    w, bias = torch.randn(N, R, generator=g).to(dtype), torch.randn(N, generator=g)
    want = torch.tanh(proj[:, off:off + R].double()) @ w.double().t() + bias.double()
    pd, wd, bd = proj.to(DEV), w.to(DEV), bias.to(DEV)
    big = torch.full((M, N + 3), 7.0, device=DEV)
    K.tanh_linear(pd[:, off:off + R], wd, bd, big[:, :N])
    _close(big[:, :N], want, 2e-5)
    assert float(big[:, N:].min()) == 7.0
    out = torch.empty(M, N, device=DEV)
    K.tanh_linear(pd[:, off:off + R], wd, None, out)
    _close(out, want - bias.double(), 2e-5)


# ------------------------------------------------------------ whole models
LENGTHS = [70, 45, 190, 33, 2, 1, 58]
TOL = {"float32": 1e-4, "bfloat16": 4e-2}       # of the largest logit


@pytest.fixture(scope="module", params=["A", "B", "C", "D"])
def model(request, tmp_path_factory):
    cfg, seed, page = C.CASES[request.param]
    folder = C.make_model(str(tmp_path_factory.mktemp(f"vufa_{request.param}")), cfg, seed,
                          drop_rank=request.param in "AC")
    reqs = {f"r{i}": H.random_ids(n, cfg["vocab"], 100 * seed + i) for i, n in enumerate(LENGTHS)}
    pc, pw = plain.load_folder(folder)
    ref = {rid: plain.forward(pc, pw, ids).float().numpy() for rid, ids in reqs.items()}
    return {"name": request.param, "cfg": cfg, "folder": folder, "page": page, "requests": reqs,
            "ref": ref, "plain": (pc, pw)}


def _bulk_tail(requests, tail):
    steps = H.trace_bulk_tail(requests, tail=tail)
    last = {}
    for st in steps:
        for e in st["entries"]:
            last[e["id"]] = st
    for rid, st in last.items():
        if rid not in st["end"]:
            st["end"].append(rid)
    return steps


def _replay(model, dtype, steps, max_tokens=None, **kw):
    from servelab_b200.replay import TraceSession
    sess = TraceSession(model["folder"], dtype, max_tokens or H.peak_tokens(steps), page_size=model["page"],
                        max_live=4, poison_cache=True, **kw)
    got = H.collect(steps, H.run_session(sess, steps), model["cfg"]["vocab"])
    sess.cache.check_invariants()
    assert not sess.held and all(p.num_free() == p.num_pages for p in sess.cache.pools)
    assert sess.cache.slots.num_free() == 4
    return got, sess


_WHOLE_BF16 = {}


def _compare(model, dtype, got):
    """float32: every position within the bound of the oracle.  bfloat16 in a model this small is
    noisy, so it is held to the oracle loosely (median and upper quartile of the error) and tightly
    to the bfloat16 logits of the same requests run WHOLE, which any schedule must reproduce up to
    the order of its sums: a fault of the cache, the state, the pages or the batch shows there."""
    scale = max(float(np.abs(r).max()) for r in model["ref"].values())
    bound = TOL[dtype] * max(1.0, scale)
    errs, first = [], None
    for rid, ids in model["requests"].items():
        assert sorted(got[rid]) == list(range(len(ids))), f"{rid}: positions missing"
        for pos in range(len(ids)):
            err = float(np.abs(got[rid][pos] - model["ref"][rid][pos]).max())
            if err > bound and first is None:
                first = (rid, pos, err)
            errs.append(err)
    errs = np.asarray(errs)
    over = int((errs > bound).sum())
    print(f"config {model['name']} {dtype}: worst abs logit error {errs.max():.3e}, median {np.median(errs):.3e}, "
          f"{over} of {len(errs)} beyond {bound:.3e} (logits up to {scale:.2f})")
    if dtype == "float32":
        assert over == 0, (f"config {model['name']}: {over} positions beyond the bound; first: request "
                           f"{first[0]} position {first[1]} (err {first[2]:.3e})")
        return
    assert np.median(errs) <= bound and np.percentile(errs, 75) <= 2.5 * bound
    whole = _WHOLE_BF16.get(model["name"])
    if whole is None:
        whole = _WHOLE_BF16[model["name"]] = _replay(model, "bfloat16", H.trace_whole(model["requests"]))[0]
    diffs = np.asarray([float(np.abs(got[rid][pos] - whole[rid][pos]).max())
                        for rid, ids in model["requests"].items() for pos in range(len(ids))])
    far = int((diffs > bound).sum())
    print(f"   against the whole prompts in bfloat16: worst {diffs.max():.3e}, {far} beyond {bound:.3e}")
    assert far <= 0.03 * len(diffs), f"{far} positions differ from the whole-prompt run"


def test_the_residual_after_every_layer_run(model):
    """The stream once a layer run's updates are added, against the oracle's: a looped layer counts each
    time it runs."""
    from servelab_b200.replay import TraceSession
    pc, pw = model["plain"]
    ids = model["requests"]["r1"]
    want = []
    plain.forward(pc, pw, ids, want)
    sess = TraceSession(model["folder"], "float32", 64, page_size=model["page"])
    seen = []
    for block in sess.runner.model.blocks:
        def fwd(ctx, resid, delta, cache, owns, _f=block.forward):
            resid, delta = _f(ctx, resid, delta, cache, owns)
            seen.append((resid + delta.materialize()).double().cpu())
            return resid, delta
        block.forward = fwd
    sess.run_step({"step": 0, "entries": [{"id": "x", "tokens": ids, "want": []}], "end": ["x"]})
    assert len(seen) == len(want) == len(plain.layer_runs(pc))
    for i, (got, ref) in enumerate(zip(seen, want)):
        assert (got - ref).abs().max() < 1e-4 * max(1.0, float(ref.abs().max())), f"layer run {i}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole(model, dtype):
    got, _ = _replay(model, dtype, H.trace_whole(model["requests"]))
    _compare(model, dtype, got)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_then_token_by_token_beyond_every_chunk(model, dtype):
    """The last 120 tokens one by one: long decoding through the state slots and the pages, with chunks
    ending among the decoded tokens."""
    got, _ = _replay(model, dtype, _bulk_tail(model["requests"], 120))
    _compare(model, dtype, got)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_down_to_two_tokens(model, dtype):
    got, _ = _replay(model, dtype, H.trace_portions(model["requests"]))
    _compare(model, dtype, got)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_with_pages_and_slots_used_again(model, dtype):
    steps = H.trace_mixed(model["requests"], seed=4)
    need = H.peak_tokens(steps)
    assert need < sum(-(-len(v) // 64) * 64 for v in model["requests"].values())
    assert len(model["requests"]) > 4                       # more requests than slots
    got, _ = _replay(model, dtype, steps, need)
    _compare(model, dtype, got)


def test_float32_logits_do_not_depend_on_the_cut(model):
    whole, _ = _replay(model, "float32", H.trace_whole(model["requests"]))
    for steps in (H.trace_portions(model["requests"]), H.trace_mixed(model["requests"], seed=9),
                  _bulk_tail(model["requests"], 40)):
        got, _ = _replay(model, "float32", steps)
        for rid in whole:
            for pos in whole[rid]:
                assert np.abs(got[rid][pos] - whole[rid][pos]).max() <= 2e-6, (rid, pos)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_single_token_steps_through_replayed_graphs(model, dtype):
    steps = _bulk_tail(model["requests"], 40)
    eager, _ = _replay(model, dtype, steps)
    graphs, sess = _replay(model, dtype, steps, cuda_graphs=True)
    assert sess.runner.graph_replays > 0
    for rid in eager:
        for pos in eager[rid]:
            assert np.abs(graphs[rid][pos] - eager[rid][pos]).max() <= (2e-6 if dtype == "float32" else 2e-1)
    _compare(model, dtype, graphs)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_steps_with_portions_through_graphs_captured_for_padded_sizes(model, dtype):
    """Steps with prompt portions replay graphs captured for padded sizes although the model keeps
    per-request state: the padding (requests without tokens, tokens of no request) must leave every
    record alone, and the warm-up run before a capture must not advance a state twice."""
    from servelab_b200.replay import TraceSession
    steps = H.trace_mixed(model["requests"], seed=4)
    eager, _ = _replay(model, dtype, steps)
    sess = TraceSession(model["folder"], dtype, H.peak_tokens(steps), page_size=model["page"], max_live=4,
                        poison_cache=True, cuda_graphs=True)
    assert sess.runner._padded_state_safe
    sess.runner.portion_graph_after = 1
    got = H.collect(steps, H.run_session(sess, steps), model["cfg"]["vocab"])
    assert sess.runner.portion_graph_replays > 0
    for rid in eager:
        for pos in eager[rid]:
            assert np.abs(got[rid][pos] - eager[rid][pos]).max() <= (2e-6 if dtype == "float32" else 2e-1), (rid, pos)
    _compare(model, dtype, got)


def test_the_trace_runner_as_a_program(model, tmp_path):
    import json
    import os
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    steps = H.trace_mixed(model["requests"], seed=21)
    out = tmp_path / "out"
    proc = subprocess.run(
        [sys.executable, os.path.join(root, "bin", "trace_run"), "--model", model["folder"], "--dtype", "bfloat16",
         "--out", str(out), "--max-tokens", str(H.peak_tokens(steps)), "--page-size", str(model["page"])],
        input="".join(json.dumps(st) + "\n" for st in steps), capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [ln for ln in proc.stdout.splitlines() if ln.startswith("done ")] == [f"done {st['step']}" for st in steps]
    V = model["cfg"]["vocab"]
    outputs = {st["step"]: np.fromfile(out / f"{st['step']}.f32", dtype="<f4").reshape(-1, V)
               for st in steps if any(e["want"] for e in st["entries"])}
    _compare(model, "bfloat16", H.collect(steps, outputs, V))


# --------------------------------------------------------------- generation
def _engine(model, dtype="float32", num_blocks=256, budget=2048, **kw):
    from servelab_b200.config import CacheConfig, SchedulerConfig
    from servelab_b200.engine.llm_engine import LLMEngine
    return LLMEngine(model["folder"], CacheConfig(block_size=model["page"], num_blocks=num_blocks),
                     SchedulerConfig(max_num_seqs=4, max_num_batched_tokens=budget), dtype=dtype, **kw)


def test_greedy_generation_through_the_engine(model):
    """The entry point and its scheduler (continuous batching, portions under a token budget,
    graphs, look-ahead) generate what the oracle generates, also with so few pages that requests
    are preempted and recomputed (their state slots start from zero again)."""
    from servelab_b200.sampling import SamplingParams
    pc, pw = model["plain"]
    prompts = [model["requests"][r][:n] for r, n in (("r0", 41), ("r1", 3), ("r2", 77), ("r5", 1), ("r3", 20))]
    n_new = 14
    want = [plain.greedy(pc, pw, p, n_new) for p in prompts]
    sp = SamplingParams(temperature=0.0, max_tokens=n_new, ignore_eos=True)
    outs = _engine(model).generate(prompts, sp)
    assert [o.outputs[0].token_ids for o in outs] == want
    outs = _engine(model, budget=16, cuda_graphs=False).generate(prompts, sp)
    assert [o.outputs[0].token_ids for o in outs] == want
    few = -(-(77 + n_new) // model["page"]) + 2
    eng = _engine(model, num_blocks=few, budget=24)
    outs = eng.generate(prompts, sp)
    assert [o.outputs[0].token_ids for o in outs] == want
    eng.runner.cache.check_invariants()
    st = eng.stats()
    assert st["running"] == 0 and st["pages_used"] == [0] * len(st["pages_used"])


def test_command_line(model, tmp_path):
    import os
    import subprocess
    import sys
    if model["name"] != "A":
        pytest.skip("one configuration is enough for the command line")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    pc, pw = model["plain"]
    want = plain.greedy(pc, pw, [3, 1, 4, 1, 5], 6)
    r = subprocess.run([sys.executable, "-m", "servelab_b200", "--model", model["folder"],
                        "--prompt-ids", "3,1,4,1,5", "--max-tokens", "6", "--temperature", "0",
                        "--dtype", "float32", "--ignore-eos", "--block-size", "8", "--num-blocks", "32"],
                       cwd=root, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert f"finish=length -> {want}" in r.stdout and "stats:" in r.stdout
