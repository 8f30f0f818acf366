"""A plain, slow implementation of the Vufadra decoder: whole sequences, float64, no cache, no
state carried between calls, one function per mechanism.  It shares no code with the package; the
tests compare the engine with it.

Notation: x [T, w] is the residual stream of one sequence, p = 0..T-1 the positions.  A layer is
x <- x + mix(shift(N1(x))) + ff(N2(x)), both read the same x (a layer without feed-forward drops
the second term), with N(u) = tanh(alpha u) * w + b element by element.  The layers
``loop.start .. loop.stop - 1`` run ``loop.times`` times in a row with the same weights, and each
pass begins with x <- W_in [x; x0] + step_t.
"""

from __future__ import annotations

import json
import math
import struct
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def _w(W, name):
    return W[name].to(F64)


# ------------------------------------------------------------------ norms
def rms_norm(x, w, eps):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def dynamic_tanh(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def _norm(x, W, name):
    return dynamic_tanh(x, _w(W, name + ".alpha"), _w(W, name), _w(W, name + ".b"))


# -------------------------------------------------------------- embedding
def bigram_rows(ids: List[int], buckets: int, mul_prev: int, mul_cur: int) -> List[int]:
    """The row of the bigram table for every token; a sequence's first token has row ``buckets``."""
    rows = []
    for t, tok in enumerate(ids):
        rows.append(buckets if t == 0 else (ids[t - 1] * mul_prev + tok * mul_cur) % buckets)
    return rows


def embed(cfg, W, ids):
    x = _w(W, "embed")[torch.tensor(ids)]
    bi = (cfg.get("embedding") or {}).get("bigram")
    if bi:
        x = x + _w(W, "bigram")[torch.tensor(bigram_rows(ids, bi["buckets"], bi["mul_prev"], bi["mul_cur"]))]
    return x


# ------------------------------------------------------------ token shift
def previous(h):
    """h of the previous token, zeros for the first."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def token_shift(h, mu):
    return h + (previous(h) - h) * mu


# --------------------------------------------------------------- rotation
def yarn_frequencies(dims: int, base: float, scaling: Optional[dict]):
    """(f_i, factor on cos and sin).  f_i = base^(-2i/dims); with ``scaling`` a ramp over i blends
    f_i (fast pairs) and f_i / factor (slow pairs)."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return torch.tensor(f, dtype=F64), 1.0
    factor, orig, fast, slow = (float(scaling[k]) for k in ("factor", "original", "fast", "slow"))

    def index_of(turns):
        return dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(index_of(fast)), 0)
    hi = min(math.ceil(index_of(slow)), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1.0 - ramp))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(factor) + 1.0


def rotate_halves(x, pos, dims: int, freq, magnitude: float = 1.0):
    """x [T, heads, D]: among the first ``dims`` elements of a head, element i turns with element
    i + dims/2 by pos * freq[i]; cos and sin are multiplied by ``magnitude``."""
    half = dims // 2
    a = pos.to(F64)[:, None] * freq[None, :]
    c, s = (torch.cos(a) * magnitude)[:, None, :], (torch.sin(a) * magnitude)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    out = x.clone()
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


# -------------------------------------------------------------- attention
def visible_in_chunk(T: int, size: int):
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    m = j <= i
    return m if not size else m & (i // size == j // size)


def sigmoid_attention(q, k, v, scale: float, bias, chunk: int):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv].  Query head h reads kv head h // (H/G);
    the weight of a visible key is sigmoid(q.k scale + bias_h), not normalized."""
    rep = q.shape[1] // k.shape[1]
    kk, vv = k.repeat_interleave(rep, dim=1), v.repeat_interleave(rep, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, kk) * scale + bias.to(F64)[:, None, None]
    p = torch.sigmoid(s) * visible_in_chunk(q.shape[0], chunk)[None].to(F64)
    return torch.einsum("hij,jhd->ihd", p, vv)


# ------------------------------------------------------------- recurrences
def delta_rule(r, k, v, w, a):
    """S_t = diag(w_t) S_{t-1} - (a_t u_t) (u_t^T S_{t-1}) + k_t v_t^T, o_t = S_t^T r_t with
    u = k / sqrt(sum k^2 + 1e-6); r, k, w, a [T, H, D], v [T, H, Dv]."""
    T, H, D = r.shape
    u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    S = torch.zeros((H, D, v.shape[-1]), dtype=F64)
    out = []
    for t in range(T):
        seen = torch.einsum("hd,hde->he", u[t], S)
        S = w[t][:, :, None] * S - (a[t] * u[t])[:, :, None] * seen[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, r[t]))
    return torch.stack(out)


def bonus_recurrence(r, k, v, w, bonus):
    """o_t = (S_{t-1} + diag(bonus) k_t v_t^T)^T r_t, then S_t = diag(w_t) S_{t-1} + k_t v_t^T;
    r, k, w [T, H, D], v [T, H, Dv], bonus [H, D]."""
    T, H, D = r.shape
    S = torch.zeros((H, D, v.shape[-1]), dtype=F64)
    out = []
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hde,hd->he", S + bonus[:, :, None] * kv, r[t]))
        S = w[t][:, :, None] * S + kv
    return torch.stack(out)


def gated_unit(u, r, i, lam):
    """log a = -8 r softplus(lam); S_t = a S_{t-1} + sqrt(1 - a^2) i u, S = 0 before the start; all
    [T, C], lam [C]."""
    log_a = -8.0 * r * torch.nn.functional.softplus(lam)
    a = torch.exp(log_a)
    gain = torch.sqrt(-torch.expm1(2.0 * log_a))
    S = torch.zeros_like(u[0])
    out = []
    for t in range(u.shape[0]):
        S = a[t] * S + gain[t] * i[t] * u[t]
        out.append(S)
    return torch.stack(out)


def short_conv(u, w, b):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_{t - taps + 1 + j} + b, zeros before the start."""
    T, C = u.shape
    taps = w.shape[1]
    pad = torch.cat([torch.zeros((taps - 1, C), dtype=F64), u])
    y = torch.zeros_like(u) + b
    for j in range(taps):
        y = y + pad[j:j + T] * w[:, j][None, :]
    return y


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ----------------------------------------------------------------- mixers
def delta_mixer(h, m: dict, W, pre: str, eps: float):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    r, k, v = ((h @ _w(W, f"{pre}.{n}").T).view(T, H, D) for n in "rkv")
    z = torch.tanh(h @ _w(W, pre + ".w1").T) @ _w(W, pre + ".w2").T + _w(W, pre + ".w0")
    w = torch.exp(-math.exp(-0.5) * torch.sigmoid(z)).view(T, H, D)
    a = torch.sigmoid(h @ _w(W, pre + ".a").T + _w(W, pre + ".a.b")).view(T, H, D)
    o = rms_norm(delta_rule(r, k, v, w, a), None, eps).reshape(T, H * D)
    return (o * _w(W, pre + ".norm") * torch.sigmoid(h @ _w(W, pre + ".g").T)) @ _w(W, pre + ".o").T


def attention_mixer(h, pos, m: dict, W, pre: str, eps: float):
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ _w(W, pre + ".q").T).view(T, H, D), _w(W, pre + ".q.norm"), eps)
    k = rms_norm((h @ _w(W, pre + ".k").T).view(T, G, D), _w(W, pre + ".k.norm"), eps)
    v = (h @ _w(W, pre + ".v").T).view(T, G, Dv)
    rot = m.get("rot")
    if rot:
        f, mag = yarn_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        q, k = rotate_halves(q, pos, rot["dims"], f, mag), rotate_halves(k, pos, rot["dims"], f, mag)
    o = sigmoid_attention(q, k, v, m["scale"], _w(W, pre + ".pb"), (m.get("mask") or {}).get("size", 0))
    return o.reshape(T, H * Dv) @ _w(W, pre + ".o").T


def time_mixer(h, m: dict, W, pre: str, eps: float):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    mixed = {s: token_shift(h, _w(W, f"{pre}.mu.{s}")) for s in "rkvgw"}
    r, k, v = ((mixed[n] @ _w(W, f"{pre}.{n}").T).view(T, H, D) for n in "rkv")
    gate = silu(mixed["g"] @ _w(W, pre + ".g").T)
    z = torch.tanh(mixed["w"] @ _w(W, pre + ".w1").T) @ _w(W, pre + ".w2").T + _w(W, pre + ".w0")
    w = torch.exp(-torch.exp(z)).view(T, H, D)
    o = rms_norm(bonus_recurrence(r, k, v, w, _w(W, pre + ".u")), None, eps).reshape(T, H * D)
    return (o * _w(W, pre + ".norm") * gate) @ _w(W, pre + ".o").T


def parallel_mixer(h, pos, m: dict, W, pre: str, eps: float):
    left = attention_mixer(h, pos, m["left"], W, pre + ".left", eps)
    right = time_mixer(h, m["right"], W, pre + ".right", eps)
    return 0.5 * (rms_norm(left, _w(W, pre + ".left.out"), eps) + rms_norm(right, _w(W, pre + ".right.out"), eps))


def block_linear(u, w, b):
    """u [T, C] in equal parts, each multiplied by a square matrix of its own: w [blocks, n, n]
    ([out, in]), b [blocks, n]."""
    T = u.shape[0]
    blocks, n, _ = w.shape
    return (torch.einsum("tbi,boi->tbo", u.view(T, blocks, n), w) + b).reshape(T, blocks * n)


def rglru_mixer(h, W, pre: str):
    y = gelu_tanh(h @ _w(W, pre + ".y").T + _w(W, pre + ".y.b"))
    u = short_conv(h @ _w(W, pre + ".x").T + _w(W, pre + ".x.b"), _w(W, pre + ".conv"), _w(W, pre + ".conv.b"))
    r = torch.sigmoid(block_linear(u, _w(W, pre + ".ra"), _w(W, pre + ".ra.b")))
    i = torch.sigmoid(block_linear(u, _w(W, pre + ".ri"), _w(W, pre + ".ri.b")))
    return (gated_unit(u, r, i, _w(W, pre + ".lam")) * y) @ _w(W, pre + ".o").T


# ----------------------------------------------------------- feed-forward
def feed_forward(h, W, pre: str):
    return (silu(h @ _w(W, pre + ".gate").T) * (h @ _w(W, pre + ".up").T)) @ _w(W, pre + ".down").T


# ------------------------------------------------------------------ model
def layer_runs(cfg: dict) -> List[tuple]:
    """(layer, pass number if the run begins a pass of the loop else None) in run order."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    out = [(i, None) for i in range(a)]
    for t in range(times):
        out += [(i, t if i == a else None) for i in range(a, b)]
    return out + [(i, None) for i in range(b, n)]


def mixer(cfg: dict, i: int, h, pos, W):
    L, pre, eps = cfg["layers"][i], f"l{i}.mix", cfg["norm"]["eps"]
    if L["type"] == "general_delta":
        return delta_mixer(h, L["mixer"], W, pre, eps)
    if L["type"] == "parallel":
        return parallel_mixer(h, pos, L["mixer"], W, pre, eps)
    if L["type"] == "rglru":
        return rglru_mixer(h, W, pre)
    raise ValueError(L["type"])


def forward(cfg: dict, W: Dict[str, torch.Tensor], ids: List[int], streams: Optional[list] = None):
    """Logits [T, vocab] float64 of one sequence; ``streams`` (a list) receives the stream after
    every layer run."""
    pos = torch.arange(len(ids))
    x = x0 = embed(cfg, W, ids)
    for i, begins in layer_runs(cfg):
        if begins is not None:
            x = torch.cat([x, x0], dim=-1) @ _w(W, "loop.in").T + _w(W, "loop.step")[begins]
        h = token_shift(_norm(x, W, f"l{i}.norm1"), _w(W, f"l{i}.shift"))
        y = mixer(cfg, i, h, pos, W)
        if cfg["layers"][i].get("mlp"):
            y = y + feed_forward(_norm(x, W, f"l{i}.norm2"), W, f"l{i}.mlp")
        x = x + y
        if streams is not None:
            streams.append(x.clone())
    return _norm(x, W, "final.norm") @ _w(W, "head").T


# ----------------------------------------------------------- model folders
_DT = {"BF16": (torch.bfloat16, 2), "F32": (torch.float32, 4), "F16": (torch.float16, 2),
       "I32": (torch.int32, 4), "I64": (torch.int64, 8)}


def read_safetensors(path: str) -> Dict[str, torch.Tensor]:
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, e in header.items():
        if name == "__metadata__":
            continue
        dt, _ = _DT[e["dtype"]]
        lo, hi = e["data_offsets"]
        out[name] = torch.frombuffer(bytearray(data[lo:hi]), dtype=dt).reshape(e["shape"]).clone()
    return out


def load_folder(folder: str):
    with open(f"{folder}/config.json") as f:
        cfg = json.load(f)
    return cfg, read_safetensors(f"{folder}/model.safetensors")


def greedy(cfg: dict, W: Dict[str, torch.Tensor], prompt: List[int], n_new: int) -> List[int]:
    """``n_new`` tokens by arg-max, the whole sequence recomputed for every token."""
    ids, out = list(prompt), []
    for _ in range(n_new):
        t = int(forward(cfg, W, ids)[-1].argmax())
        out.append(t)
        ids.append(t)
    return out
