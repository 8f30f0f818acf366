"""Sunutar on the GPU against the plain implementation (``plain_sunutar``): every new mechanism alone, then whole
models replayed whole, token by token, in portions down to two tokens and in mixed batches with pages and
slots used again, in float32 and bfloat16, and greedy generation through the engine."""

import numpy as np
import pytest
import torch

import helpers as H
import plain_sunutar as plain
import sunutar_cases as C

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


# -------------------------------------------- norms before and after a sublayer
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("w", [4, 48, 50, 1028, 2048, 16500])
def test_norm_of_the_result_add_and_next_norm(dtype, w):
    """One launch: the update's norm (with its factor in the weight), the add, the next norm; selected rows leave
    the stream as it is; an update as partial sums with a bias."""
    from servelab_b200.ops import kernels as K
    g = torch.Generator().manual_seed(w)
    T = 7
    resid, upd = torch.randn(T, w, generator=g) * 3, (torch.randn(T, w, generator=g) * 20).to(dtype)
    pw, nw = torch.randn(w, generator=g), torch.randn(w, generator=g)
    x = resid.double() + plain.rms_norm(upd.double(), pw.double(), 1e-3)
    want = plain.rms_norm(x, nw.double(), 1e-5)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    r, u, p, n = resid.to(DEV), upd.to(DEV), pw.to(DEV), nw.to(DEV)
    rows = torch.tensor([3, 0, 6], dtype=torch.int32, device=DEV)
    out = torch.empty(3, w, dtype=dtype, device=DEV)
    K.post_add_rmsnorm(r, u, p, 1e-3, n, 1e-5, out, rows)
    _close(out, want[[3, 0, 6]], tol)
    assert torch.equal(r.cpu(), resid)
    out = torch.empty(T, w, dtype=dtype, device=DEV)
    K.post_add_rmsnorm(r, u, p, 1e-3, n, 1e-5, out)
    _close(out, want, tol)
    _close(r, x, 1e-5)
    parts, bias = torch.randn(3, T, w, generator=g), torch.randn(w, generator=g)
    total = parts.double().sum(0) + bias.double()
    x = resid.double() + plain.rms_norm(total, pw.double(), 1e-3)
    r = resid.to(DEV)
    K.post_add_rmsnorm(r, K.SplitSum(parts.to(DEV), bias.to(DEV), dtype), p, 1e-3, n, 1e-5, out)
    _close(out, plain.rms_norm(x, nw.double(), 1e-5), tol)
    _close(r, x, 1e-5 if dtype == torch.float32 else 1e-4)


def test_a_small_update_counts_in_full_and_eps_sits_inside_the_root():
    from servelab_b200.ops import kernels as K
    resid = torch.zeros(2, 64, device=DEV)
    upd = torch.full((2, 64), 1e-3, device=DEV)
    upd[1] = 1e-6
    one, out = torch.ones(64, device=DEV), torch.empty(2, 64, device=DEV)
    K.post_add_rmsnorm(resid, upd, one, 1e-6, one, 1e-12, out)
    want = torch.tensor([1e-3 / (1e-6 + 1e-6) ** 0.5, 1e-6 / (1e-12 + 1e-6) ** 0.5])
    assert torch.allclose(resid[:, 0].cpu(), want, rtol=1e-5)


# -------------------------------------- biases, norms over whole rows, cache write
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("shape", [(4, 2, 16, 8), (3, 1, 10, 6), (16, 4, 128, 64), (1, 1, 64, 64), (6, 6, 40, 24)])
@pytest.mark.parametrize("many", [False, True])
def test_head_kernel_with_biases_and_row_norms(dtype, shape, many):
    """Keys and values go to their pages, the query heads of a token are normed together and so are its key heads,
    biases first; columns of a wider row."""
    from servelab_b200.ops import kernels as K
    Hq, G, D, Dv = shape
    ps = 8
    T = 530 if many else 21
    g = torch.Generator().manual_seed(D)
    qs, ks, vs = Hq * D, G * D, G * Dv
    wide = (torch.randn(T, qs + ks + vs + 24, generator=g) * torch.linspace(0.2, 3.0, qs + ks + vs + 24)).to(dtype)
    qb, kb, vb = (torch.randn(n, generator=g) for n in (qs, ks, vs))
    qw, kw = torch.randn(qs, generator=g), torch.randn(ks, generator=g)
    n_pages = -(-T // ps) + 2
    table = torch.randperm(n_pages, generator=g).tolist()
    ctx = _ctx([_entry(T, 0, table[:-(-T // ps)])])
    kc, vc = (torch.zeros(n_pages, G, ps, d, dtype=dtype, device=DEV) for d in (D, Dv))
    q = torch.empty(T, qs, dtype=dtype, device=DEV)
    proj = wide.to(DEV)[:, 16:]
    K.head_prep(proj, ctx, ctx.block_tables[0], ps, q_off=0, num_heads=Hq, q_dim=D, q_norm_w=qw.to(DEV), q_norm_dims=0,
                q_rot_off=0, k_off=qs, num_kv_heads=G, k_dim=D, k_norm_w=kw.to(DEV), k_norm_dims=0, k_rot_off=0,
                v_off=qs + ks, v_dim=Dv, freq=None, rot_dims=0, rot_mag=1.0, eps=1e-4, q_out=q, k_cache=kc, v_cache=vc,
                q_bias=qb.to(DEV), k_bias=kb.to(DEV), v_bias=vb.to(DEV), row_norm=True)
    p = wide[:, 16:].double()
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    _close(q, plain.rms_norm(p[:, :qs] + qb, qw.double(), 1e-4), tol, "q")
    k = plain.rms_norm(p[:, qs:qs + ks] + kb, kw.double(), 1e-4).view(T, G, D)
    v = (p[:, qs + ks:qs + ks + vs] + vb).view(T, G, Dv)
    at = torch.tensor([table[t // ps] for t in range(T)])
    slot = torch.arange(T) % ps
    _close(kc.cpu()[at, :, slot], k, tol, "k")
    _close(vc.cpu()[at, :, slot], v, tol, "v")
    assert K.head_prep_status() == 0


# --------------------------------- attention: distance bias, cap, window, the added one
def _attention_case(seed, Hq, G, Dk, Dv, window, ctxs, qlens, ps, dtype, spike, scale, cap):
    """Requests with contexts ``ctxs`` whose last ``qlens`` tokens are this step's queries; keys and values in
    pages in a shuffled order (unwritten slots hold a huge number).  ``spike`` "in" / "out": for every query the
    last key inside its window / the first outside it stands out (marked keys every ``window``, which some query
    meets at either edge); "far": the first key of the request does."""
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
            q[..., 0] = 3.0                            # what the marked keys answer to ...
            k[..., 0] = -4.0                           # ... and the others do not
            at = {"far": [0], "in": [max(0, c - (window or c))], "out": [max(0, c - (window or c) - 1)]}[spike]
            if window and n > 1:
                at = list(range(at[0] % window, c, window))
            k[at, :, 0] = 6.0
            v[at] = 7.0
        k, v, q = k.to(dtype), v.to(dtype), q.to(dtype)
        table = [order.pop() for _ in range(-(-c // ps))]
        for p in range(c):
            kc[table[p // ps], :, p % ps] = k[p]
            vc[table[p // ps], :, p % ps] = v[p]
        if window:                                     # pages behind every query's window have gone back
            for lp in range(max(0, c - n - window + 1) // ps):
                kc[table[lp]], vc[table[lp]] = 1e30, 1e30
                table[lp] = -1
        qfull = torch.zeros(c, Hq, Dk, dtype=F64)
        qfull[c - n:] = q.double()
        o = plain.distance_attention(qfull, k.double(), v.double(), scale, cap, window)
        wants.append(o[c - n:].reshape(n, Hq * Dv))
        qs.append(q.reshape(n, Hq * Dk))
        entries.append(_entry(n, c - n, table))
    return {"q": torch.cat(qs).to(DEV), "kc": kc.to(DEV), "vc": vc.to(DEV), "want": torch.cat(wants), "entries": entries}


# heads, kv heads, key and value size, window, cap
SHAPES = [(4, 2, 80, 48, None, 6.0), (5, 1, 112, 96, 40, 20.0), (3, 3, 10, 6, 9, 8.0), (8, 2, 64, 64, 90, 12.0),
          (6, 1, 128, 128, 1, 5.0), (4, 2, 32, 32, 33, None), (2, 1, 160, 128, 300, 30.0), (16, 2, 64, 128, 70, 9.0),
          (1, 1, 64, 64, 64, None), (34, 2, 16, 16, 128, 10.0), (12, 12, 64, 64, None, 15.0)]


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("spike", ["in", "out", "far", None])
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("decode", [False, True])
def test_attention_with_a_distance_bias(dtype, spike, shape, decode):
    """Portions and single tokens at page, tile and window edges, the first token alone (whose weight is
    e^s / (1 + e^s)), results times a factor into columns of a wider row that is not touched elsewhere."""
    from servelab_b200.ops import attention as A
    from servelab_b200.ops import kernels as K
    Hq, G, Dk, Dv, window, cap = shape
    ps, factor = 8, 0.625
    w = window or 64
    ctxs = [1, 2, 300, 301, 64, 65, 333, w, w + 1, 2 * w, 2 * w + 1]
    qlens = [1] * len(ctxs) if decode else [1, 2, 200, 37, 64, 3, 33, w, 2, w + 1, 1]
    case = _attention_case(7, Hq, G, Dk, Dv, window, ctxs, qlens, ps, dtype, spike, 0.3, cap)
    slopes = plain.head_slopes(Hq).float().to(DEV)
    zero = torch.zeros(Hq, device=DEV)
    ctx = _ctx(case["entries"])

    def run():
        row = torch.full((case["q"].shape[0], Hq * Dv + 16), 9.0, dtype=dtype, device=DEV)
        out = row[:, :Hq * Dv]
        A.kv_attention(ctx, case["q"], case["kc"], case["vc"], Dv, out, ctx.block_tables[0], Hq, G, Dk, Dv,
                       ps, 0.3, window or 0, None, cap, zero, slopes=slopes, out_scale=factor)
        assert float((row[:, Hq * Dv:] - 9.0).abs().max()) == 0
        return out
    tol = 1e-5 if dtype == torch.float32 else 1.5e-2
    want = case["want"] * factor
    _close(run(), want, tol)
    if dtype == torch.bfloat16:
        A.force_generic = True                         # the plain kernel is the twin of the tensor-core ones ...
        try:
            _close(run(), want, tol, "plain")
        finally:
            A.force_generic = False
        A.use_kv_tc_capped = False                     # ... and mma.sync the twin of tcgen05
        try:
            _close(run(), want, tol, "mma")
        finally:
            A.use_kv_tc_capped = True
        if decode:                                     # ... as are the two forms for single tokens
            saved = K.attention_kv_warp_keys_min
            try:
                for least in (0, 1 << 30):
                    K.attention_kv_warp_keys_min = least
                    _close(run(), want, tol, least)
            finally:
                K.attention_kv_warp_keys_min = saved
        if Dk % 64 == 0 and Dv % 64 == 0:
            assert K.attention_kv_tc_status(Dk, Dv) == 0 and K.attention_kv_mma_status(Dk, Dv) == 0


@pytest.mark.parametrize("window,ctxs", [(None, [1500, 900, 1]), (1100, [1100, 2201, 900])])
@pytest.mark.parametrize("least", [0, 1 << 30])
@pytest.mark.parametrize("shape", [(8, 2, 64, 48, 16), (12, 1, 192, 256, 8), (3, 1, 128, 128, 32)])
def test_attention_single_tokens_with_key_splits_and_a_distance_bias(window, ctxs, least, shape, monkeypatch):
    """Few requests with long contexts: the keys are split over blocks; the added one counts once.  Both forms of the
    kernel."""
    from servelab_b200.ops import attention as A
    from servelab_b200.ops import kernels as K
    monkeypatch.setattr(K, "attention_kv_warp_keys_min", least)
    Hq, G, Dk, Dv, ps = shape
    for spike in ("in", "far", None):
        case = _attention_case(5, Hq, G, Dk, Dv, window, ctxs, [1, 1, 1], ps, torch.bfloat16, spike, 0.3, 14.0)
        ctx = _ctx(case["entries"])
        out = torch.empty(3, Hq * Dv, dtype=torch.bfloat16, device=DEV)
        A.kv_attention(ctx, case["q"], case["kc"], case["vc"], Dv, out, ctx.block_tables[0], Hq, G, Dk, Dv, ps, 0.3,
                       window or 0, None, 14.0, torch.zeros(Hq, device=DEV), slopes=plain.head_slopes(Hq).float().to(DEV),
                       out_scale=1.5)
        _close(out, case["want"] * 1.5, 1.5e-2, spike)


@pytest.mark.parametrize("chunk", [0, 700])
def test_single_token_forms_agree_on_gates_sigmoid_weights_and_tied_values(chunk, monkeypatch):
    """What other designs ask of the kernel for single tokens: weights that are not normalized in chunks, a gate a
    head, values that are a prefix of the keys, a learned sink -- the two forms against each other."""
    from servelab_b200.ops import attention as A
    from servelab_b200.ops import kernels as K
    Hq, G, Dk, Dv, ps = 6, 2, 96, 64, 16
    case = _attention_case(9, Hq, G, Dk, Dv, None, [1400, 650, 40], [1, 1, 1], ps, torch.bfloat16, None, 0.2, None)
    ctx = _ctx(case["entries"])
    gate = torch.randn(3, Hq, device=DEV).to(torch.bfloat16)
    extra = torch.linspace(-2.0, 2.0, Hq, device=DEV)

    def run(least, tied, **kw):
        monkeypatch.setattr(K, "attention_kv_warp_keys_min", least)
        out = torch.empty(3, Hq * Dv, dtype=torch.bfloat16, device=DEV)
        v = case["kc"] if tied else case["vc"]
        A.kv_attention(ctx, case["q"], case["kc"], v, Dk if tied else Dv, out, ctx.block_tables[0], Hq, G, Dk, Dv, ps, 0.2,
                       0, **kw)
        return out.double().cpu()
    for tied in (False, True):
        for kw in (dict(head_gate=gate, chunk=chunk), dict(head_gate=gate, sink=extra, softcap=5.0, chunk=chunk),
                   dict(head_gate=None, sigmoid_bias=extra, chunk=chunk)):
            a, b = run(0, tied, **kw), run(1 << 30, tied, **kw)
            assert (a - b).abs().max() < 1e-2 * max(1.0, float(b.abs().max())), (tied, list(kw))


# ------------------------------------------------------- convolution with SiLU
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("C_,taps", [(64, 3), (50, 4), (1024, 2), (24, 1), (40, 5)])
def test_convolution_with_bias_and_silu(dtype, C_, taps):
    """Whole, in portions and token by token; columns of a wider projection, the record a slice of a larger one
    that keeps the rows before the activation."""
    from servelab_b200.ops import kernels as K
    g = torch.Generator().manual_seed(C_)
    n, m = 30, 9
    wide = torch.randn(n + m, C_ + 16, generator=g).to(dtype)
    w, b = torch.randn(C_, taps, generator=g) * 0.5, torch.randn(C_, generator=g)
    x = wide[:, 8:8 + C_].double()
    want = torch.cat([plain.silu(plain.short_conv(x[s], w.double(), b.double())) for s in (slice(0, n), slice(n, n + m))])
    wd, tw, bd = wide.to(DEV), w.t().contiguous().to(DEV), b.to(DEV)
    for name, schedule in _schedules(n, m).items():
        big = torch.full((3, (taps - 1) * C_ + 8), 3.0, device=DEV)
        state = big[:, 4:4 + (taps - 1) * C_] if taps > 1 else None
        zeroed = state if state is not None else torch.zeros(3, 1, device=DEV)

        def body(rows, ctx):
            out = torch.empty(len(rows), C_, dtype=dtype, device=DEV)
            K.short_conv(wd[rows].contiguous()[:, 8:], tw, state, ctx, out, None, bd, activation="silu")
            return out
        _close(_run(schedule, zeroed, body, n), want, 1e-5 if dtype == torch.float32 else 1e-2, name)
        if taps > 1:
            _close(state[0], x[n - taps + 1:n].reshape(-1), 1e-6)
            assert float(big[:, :4].min()) == 3.0 and float(big[:, -4:].min()) == 3.0


# ------------------------------------------------------------ state space
# heads, value size, state, groups
SPACES = [(3, 16, 8, 1), (2, 48, 64, 2), (1, 64, 128, 1), (4, 64, 64, 2), (3, 7, 9, 3), (6, 80, 144, 3), (5, 24, 48, 5),
          (2, 130, 256, 1), (1, 200, 33, 1), (8, 32, 16, 4)]


def _space_case(seed, shape, T, dtype, slow):
    Hh, P, N, G = shape
    g = torch.Generator().manual_seed(seed)
    u = torch.randn(T, Hh * P + 2 * G * N, generator=g).to(dtype)
    dt = torch.randn(T, Hh, generator=g) * 2 - (4.0 if slow else 0.0)
    return u, dt, torch.randn(Hh, generator=g), torch.randn(Hh, generator=g) * 1.5 - (3.0 if slow else 0.0), torch.randn(Hh, generator=g)


def _space_want(case, shape, lens):
    Hh, P, N, G = shape
    u, dt, bias, a_log, skip = (t.double() for t in case)
    outs = []
    for a, b in lens:
        n, inner = b - a, Hh * P
        x, B, Cc = u[a:b, :inner].view(n, Hh, P), u[a:b, inner:inner + G * N].view(n, G, N), u[a:b, inner + G * N:].view(n, G, N)
        d = torch.nn.functional.softplus(dt[a:b] + bias, threshold=1e9)
        outs.append(plain.selective_recurrence(x, B, Cc, d, a_log, skip).reshape(n, inner))
    return torch.cat(outs)


def _run_space(K, case, shape, rows, ctx, state):
    Hh, P, N, G = shape
    u, dt, bias, a_log, skip = case
    out = torch.empty(len(rows), Hh * P, dtype=torch.float32, device=DEV)
    K.state_space(ctx, u[rows].contiguous(), dt[rows].contiguous(), state, out, num_heads=Hh, value_dim=P, state_dim=N,
                  groups=G, dt_bias=bias, rate=torch.exp(a_log), skip=skip)
    return out


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("shape", SPACES)
@pytest.mark.parametrize("slow", [False, True])
def test_state_space_token_by_token(dtype, shape, slow, monkeypatch):
    """Whole, in portions and token by token, bit for bit the same; the record may be a slice of a larger one."""
    from servelab_b200.ops import kernels as K
    monkeypatch.setattr(K, "state_space_chunked", False)
    Hh, P, N, G = shape
    n, m = 41, 7
    host = _space_case(3, shape, n + m, dtype, slow)
    want = _space_want(host, shape, [(0, n), (n, n + m)])
    case = tuple(t.to(DEV) for t in host)
    rec = Hh * P * N
    results = []
    for name, schedule in _schedules(n, m).items():
        big = torch.full((3, -(-rec // 4) * 4 + 8), 3.0, device=DEV)
        state = big[:, 4:4 + rec]
        got = _run(schedule, state, lambda rows, ctx: _run_space(K, case, shape, rows, ctx, state), n)
        _close(got, want, 3e-5, name)
        assert float(big[:, :4].min()) == 3.0 and float(big[:, 4 + rec:].min()) == 3.0
        results.append((got, state[[0, 2]].clone()))
    for got, st in results[1:]:
        assert torch.equal(got, results[0][0]) and torch.equal(st, results[0][1])
    keep = state.clone()
    u, dt = case[0][:16], case[1][:16]
    _run_space(K, (u, dt) + case[2:], shape, torch.arange(16), _padded_ctx([_entry(2, 0, (), 1)], 16, 2), state)
    assert torch.equal(state[[0, 2]], keep[[0, 2]]) and not torch.equal(state[1], keep[1])


@pytest.mark.parametrize("shape", SPACES)
@pytest.mark.parametrize("slow", [False, True])
def test_state_space_in_chunks(shape, slow, monkeypatch):
    """The chunked kernels: requests shorter than a chunk, a chunk exactly, a chunk and one token, several chunks,
    cuts inside chunks, the state they leave against the token-by-token kernel's, padding."""
    from servelab_b200.ops import kernels as K
    monkeypatch.setattr(K, "state_space_chunk_min_tokens", 1)
    Hh, P, N, G = shape
    lens, starts = [5, 64, 65, 300], [0, 5, 69, 134]
    T = sum(lens)
    host = _space_case(11, shape, T, torch.bfloat16, slow)
    want = _space_want(host, shape, [(a, a + k) for a, k in zip(starts, lens)])
    case = tuple(t.to(DEV) for t in host)
    rec = Hh * P * N
    big = torch.full((4, -(-rec // 4) * 4 + 8), 3.0, device=DEV)
    state = big[:, 4:4 + rec]
    state.zero_()

    def step(pieces):
        rows = torch.cat([torch.arange(a, a + k) for _, a, k in pieces])
        ctx = _ctx([_entry(k, 0, (), slot) for slot, a, k in pieces], 0)
        return rows, _run_space(K, case, shape, rows, ctx, state)
    tol = 1e-4
    _, got = step([(s, a, k) for s, (a, k) in enumerate(zip(starts, lens))])
    _close(got, want, tol)
    assert float(big[:, :4].min()) == 3.0 and float(big[:, 4 + rec:].min()) == 3.0
    final = state.clone()
    state.zero_()
    a = 134
    for k in (90, 16, 128, 2, 64):
        rows, got = step([(3, a, k)])
        _close(got, want[rows], tol, a)
        a += k
    _close(state[3], final[3].double().cpu(), tol, "cut")
    state.zero_()
    monkeypatch.setattr(K, "state_space_chunked", False)
    step([(3, 134, 300)])
    _close(state[3], final[3].double().cpu(), tol, "token by token")
    monkeypatch.setattr(K, "state_space_chunked", True)
    keep = state.clone()
    _run_space(K, case, shape, torch.arange(48), _padded_ctx([_entry(40, 0, (), 1)], 48, 2), state)
    assert torch.equal(state[[0, 2, 3]], keep[[0, 2, 3]]) and not torch.equal(state[1], keep[1])


def test_state_space_remembers_and_forgets():
    """One input 1,500 tokens back, asked for by the last token: a head that does not decay still answers with
    d x, one that decays slowly has the closed form's share, a fast one nothing; in chunks, token by token, both."""
    from servelab_b200.ops import kernels as K
    shape = (3, 8, 16, 1)
    Hh, P, N, G = shape
    T = 1501
    u = torch.zeros(T, Hh * P + 2 * N)
    u[0, :Hh * P] = torch.arange(1.0, 9.0).repeat(3)
    u[0, Hh * P + 5] = 1.0                                       # B_0 = e_5
    u[T - 1, Hh * P + N + 5] = 2.0                               # C_last = 2 e_5
    dt = torch.zeros(T, Hh)                                      # d = ln 2
    a_log = torch.tensor([-40.0, -7.0, 0.0])
    case = tuple(t.to(DEV) for t in (u.to(torch.bfloat16), dt, torch.zeros(Hh), a_log, torch.zeros(Hh)))
    x, d = torch.arange(1.0, 9.0, dtype=F64), np.log(2.0)
    for cuts in ([T], [1] * T, [700, 1, 30, 70, 700]):
        state = torch.zeros(1, Hh * P * N, device=DEV)
        a = 0
        for k in cuts:
            out = _run_space(K, case, shape, torch.arange(a, a + k), _ctx([_entry(k, a)], 0), state)
            a += k
        last = out[-1].double().cpu().view(Hh, P)
        assert (last[0] - 2 * d * x).abs().max() < 1e-4
        assert (last[1] - 2 * d * x * np.exp(-np.exp(-7.0) * d * 1500)).abs().max() < 2e-4
        assert last[2].abs().max() == 0


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("n,groups", [(48, 4), (50, 1), (21, 7), (2048, 1), (4096, 2), (6144, 2), (96, 96)])
def test_gate_before_the_norm_of_parts(dtype, n, groups):
    from servelab_b200.ops import kernels as K
    g = torch.Generator().manual_seed(n)
    T = 9
    y = torch.randn(T, n, generator=g) * torch.linspace(0.1, 5.0, n)
    z = torch.randn(T, n + 8, generator=g).to(dtype)
    w = torch.randn(n, generator=g)
    want = 0.7 * plain.gated_group_norm(y.double(), z[:, :n].double(), w.double(), groups, 1e-3)
    row = torch.full((T, n + 16), 9.0, dtype=dtype, device=DEV)
    K.gate_group_norm(y.to(DEV), z.to(DEV), groups, row[:, 8:8 + n], eps=1e-3, weight=w.to(DEV), factor=0.7)
    _close(row[:, 8:8 + n], want, 1e-5 if dtype == torch.float32 else 1e-2)
    assert float(row[:, :8].min()) == 9.0 and float(row[:, 8 + n:].min()) == 9.0


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
def test_parallel_mixer_alone(dtype, which):
    """Both branches through the merged products against the oracle's mixer, in three schedules, every layer of
    a configuration."""
    from servelab_b200.config import config_from_dict
    from servelab_b200.ops.kernels import plain_unless
    from servelab_b200.parts import BuildEnv, LayerCache
    from servelab_b200.parts.parallel_mixers import ParallelMixers
    from servelab_b200.weights import RandomSource
    cfg = C.CASES[which][0]
    n, m, ps = 75, 9, 8
    for i, b in enumerate(config_from_dict(cfg).to_model_spec().layers):
        spec = b.mixer
        src = RandomSource(ParallelMixers.declare(spec, f"l{i}.mix"), 3, std=0.15, norm_std=0.3, dtype=torch.bfloat16,
                           std_of=C.STD_OF)
        W = {name: src.read(name) for name in src.names()}
        matrices = {f"l{i}.mix.{x}" for x in ("left.q", "left.k", "left.v", "left.o", "right.in", "right.o")}

        class Store:
            def get(self, name):
                return W[name].to(DEV, dtype if name in matrices else torch.float32).contiguous()

            def cat(self, names):
                return torch.cat([self.get(x) for x in names])
        mixer = ParallelMixers(spec, f"l{i}.mix", BuildEnv(device=DEV, dtype=dtype, page_size=ps))
        mixer.load(Store())
        g = torch.Generator().manual_seed(i)
        x = torch.randn(n + m, cfg["width"], generator=g).to(dtype)
        want = torch.cat([plain.parallel_mixer(x[s].double(), cfg["layers"][i]["mixer"], W, f"l{i}.mix", cfg["norm"]["eps"])
                          for s in (slice(0, n), slice(n, n + m))])
        xd = x.to(DEV)
        floats = sum(mixer.sizes)
        pages = -(-n // ps) + -(-m // ps)
        tables = {0: list(range(-(-n // ps))), 2: list(range(-(-n // ps), pages))}
        for name, schedule in _schedules(n, m).items():
            kc = torch.full((pages, spec.left.num_kv_heads, ps, spec.left.head_dim), 1e30, dtype=dtype, device=DEV)
            vc = torch.full((pages, spec.left.num_kv_heads, ps, spec.left.value_dim), 1e30, dtype=dtype, device=DEV)
            state = torch.full((3, floats), 3.0, device=DEV)
            outs = {}
            for step in schedule:
                for slot, a, k in step:
                    if a in (0, n):
                        state[slot].zero_()
                rows = torch.cat([torch.arange(a, a + k) for _, a, k in step])
                ctx = _ctx([_entry(k, a - (0 if a < n else n), tables[slot], slot) for slot, a, k in step])
                y = plain_unless(None, mixer.forward(ctx, xd[rows].contiguous(),
                                                     LayerCache(group=0, k=kc, v=vc, state=state, page_size=ps), True))
                for r, row in zip(rows.tolist(), y):
                    outs[r] = row
            got = torch.stack([outs[r] for r in sorted(outs)])
            # (a norm part of few elements divides by a small root mean square now and then)
            _close(got, want, 1e-4 if dtype == torch.float32 else 8e-2, (which, i, name))
            assert float(state[1].min()) == 3.0


# ---------------------------------------------------------------- experts
def test_router_takes_the_largest_sigmoids_and_keeps_them():
    from servelab_b200.ops import kernels as K
    g = torch.Generator().manual_seed(2)
    for E, top in ((5, 2), (1, 1), (64, 7), (300, 32), (3, 3)):
        z = torch.randn(77, E, generator=g) * 3
        z[5] = 0.25                                    # ties: the lower index
        z[6] = torch.randperm(E, generator=g) / 64.0 + 25.0     # sigmoids that round to 1 in float32
        ids, w = K.moe_route_scored(z.to(DEV), 1, 1, top, 1.0, False, "sigmoid")
        wi, ww = plain.route(z.double(), top)
        assert torch.equal(ids.cpu().long(), wi)
        _close(w, ww, 1e-6)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("shape", [(40, 48, 24, 5, 2), (70, 50, 14, 3, 3), (1, 64, 64, 1, 1), (200, 128, 64, 9, 1),
                                   (600, 2048, 1024, 3, 2)])
def test_experts_weighted_at_their_inputs(dtype, shape):
    """The clamped activation is not linear, so a weight at the output would differ; the large shape takes the
    library's grouped product in bfloat16."""
    from servelab_b200.ops import kernels as K
    T, h, ff, E, top = shape
    if dtype == torch.float32 and h > 1000:
        pytest.skip("the large shape is there for the grouped product")
    g = torch.Generator().manual_seed(h)
    x = torch.randn(T, h, generator=g).to(dtype)
    W = {}
    for e in range(E):
        for n, s in (("gate", (ff, h)), ("up", (ff, h)), ("down", (h, ff))):
            W[f"m.e{e}.{n}"] = (torch.randn(s, generator=g) * (2.0 / s[1] ** 0.5)).to(dtype)
    ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)])
    wgt = torch.rand(T, top, generator=g) * 0.9 + 0.05
    want = torch.zeros(T, h, dtype=F64)
    for e in range(E):
        t, k = torch.where(ids == e)
        want[t] += plain.dense(wgt[t, k].double()[:, None] * x[t].double(), W, f"m.e{e}", 1.3)
    gu = torch.stack([torch.cat([W[f"m.e{e}.gate"], W[f"m.e{e}.up"]]) for e in range(E)]).to(DEV)
    dn = torch.stack([W[f"m.e{e}.down"] for e in range(E)]).to(DEV)
    args = (x.to(DEV), ids.to(torch.int32).to(DEV), wgt.to(DEV), gu, dn, None, "swish_clamped", 1.3, 1.702, True)
    tol = 1e-5 if dtype == torch.float32 else 2e-2
    _close(K.moe_experts(*args), want, tol)
    if dtype == torch.bfloat16:
        K.moe_vendor_grouped = False
        try:
            _close(K.moe_experts(*args), want, tol, "own products")
            K.moe_tensor_cores = False
            _close(K.moe_experts(*args), want, tol, "CUDA cores")
        finally:
            K.moe_vendor_grouped = K.moe_tensor_cores = True


@pytest.mark.parametrize("dtype", BOTH)
def test_gated_activation_with_a_factor_a_row(dtype):
    from servelab_b200.ops import kernels as K
    g = torch.Generator().manual_seed(4)
    for T, n in ((5, 64), (3, 20), (4, 7)):
        gu, rs = torch.randn(T, 2 * n, generator=g).to(dtype), torch.rand(T, generator=g)
        out = torch.empty(T, n, dtype=dtype, device=DEV)
        K.gated_act(gu.to(DEV), out, 0, "swish_clamped", 0.8, 1.702, rs.to(DEV))
        s = gu.double() * rs.double()[:, None]
        _close(out, plain.clamped_unit(s[:, :n], s[:, n:], 0.8), 1e-5 if dtype == torch.float32 else 1e-2)


# ------------------------------------------------------------ whole models
LENGTHS = [70, 45, 190, 33, 2, 1, 58]
TOL = {"float32": 1e-4, "bfloat16": 4e-2}       # of the largest logit


@pytest.fixture(scope="module", params=["A", "B", "C", "D"])
def model(request, tmp_path_factory):
    cfg, seed, page = C.CASES[request.param]
    folder = C.make_model(str(tmp_path_factory.mktemp(f"sunu_{request.param}")), cfg, seed)
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


def _same(model, dtype, got, want):
    """Two runs of the same steps, to rounding (a router's close call may fall the other way in bfloat16)."""
    scale = max(float(np.abs(r).max()) for r in model["ref"].values())
    diffs = np.asarray([float(np.abs(got[rid][pos] - want[rid][pos]).max()) for rid in want for pos in want[rid]])
    if dtype == "float32":
        assert diffs.max() <= 2e-6 * scale
    else:
        assert (diffs > 1e-2 * scale).sum() <= 0.03 * len(diffs)


def test_the_residual_after_every_layer(model):
    """The stream once a layer's updates are added, against the oracle's."""
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
    assert len(seen) == len(want) == len(pc["layers"])
    for i, (got, ref) in enumerate(zip(seen, want)):
        assert (got - ref).abs().max() < 1e-4 * max(1.0, float(ref.abs().max())), f"layer {i}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole(model, dtype):
    got, _ = _replay(model, dtype, H.trace_whole(model["requests"]))
    _compare(model, dtype, got)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_then_token_by_token_beyond_every_window(model, dtype):
    """The last 120 tokens one by one: long decoding through the state slots and the pages, with windows
    passing over decoded tokens."""
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
    _same(model, dtype, graphs, eager)
    _compare(model, dtype, graphs)


def test_branches_on_two_streams_equal_one_stream(model, monkeypatch):
    """Captured steps run the two branches side by side; bit for bit the results of one stream."""
    from servelab_b200.parts import parallel_mixers as PM
    steps = H.trace_mixed(model["requests"], seed=4)
    from servelab_b200.replay import TraceSession
    got = []
    for overlap in (True, False, True):
        monkeypatch.setattr(PM, "overlap_branches", overlap)
        sess = TraceSession(model["folder"], "bfloat16", H.peak_tokens(steps), page_size=model["page"], max_live=4,
                            poison_cache=True, cuda_graphs=True)
        sess.runner.portion_graph_after = 1
        got.append(H.collect(steps, H.run_session(sess, steps), model["cfg"]["vocab"]))
        assert sess.runner.portion_graph_replays > 0
    for rid in got[0]:
        for pos in got[0][rid]:
            assert np.array_equal(got[0][rid][pos], got[1][rid][pos]) and np.array_equal(got[0][rid][pos], got[2][rid][pos])


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
    _same(model, dtype, got, eager)
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
