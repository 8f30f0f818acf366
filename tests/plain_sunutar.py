"""A plain, slow implementation of the Sunutar decoder: whole sequences, float64, no cache, no state
carried between calls, one function per mechanism.  It shares no code with the package; the tests
compare the engine with it.

Notation: x [T, w] is the residual stream of one sequence.  A layer is x <- x + m N1b(mix(N1(x))),
then x <- x + m N2b(ff(N2(x))) (a layer without feed-forward ends after the first half), with RMS
norms and one factor m for the model.
"""

from __future__ import annotations

import json
import struct
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def _w(W, name):
    return W[name].to(F64)


def rms_norm(x, w, eps):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(z):
    return z * torch.sigmoid(z)


# -------------------------------------------------------------- attention
def head_slopes(heads: int):
    """slope_h = 2^(-8 (h + 1) / heads)."""
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=F64)


def visible(T: int, window: Optional[int]):
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    m = j <= i
    return m if not window else m & (i - j < window)


def distance_attention(q, k, v, scale: float, cap: Optional[float], window: Optional[int]):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv].  Query head h reads kv head h // (H/G); a
    scaled score s becomes cap tanh(s / cap) - slope_h (i - j); the weights are exp(s) / (1 + sum exp(s))."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    kk, vv = k.repeat_interleave(rep, dim=1), v.repeat_interleave(rep, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, kk) * scale
    if cap:
        s = cap * torch.tanh(s / cap)
    dist = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).to(F64)
    s = s - head_slopes(H)[:, None, None] * dist[None]
    s = s.masked_fill(~visible(T, window)[None], -torch.inf)
    top = s.amax(-1, keepdim=True).clamp(min=0.0)          # (the added one is exp(0))
    e = torch.exp(s - top)
    p = e / (torch.exp(-top) + e.sum(-1, keepdim=True))
    return torch.einsum("hij,jhd->ihd", p, vv)


def attention_mixer(h, m: dict, W, pre: str, eps: float):
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ _w(W, f"{pre}.{n}").T + _w(W, f"{pre}.{n}.b") for n in "qkv")
    q = rms_norm(q, _w(W, pre + ".q.norm"), eps).view(T, H, D)     # the whole row, before it is split
    k = rms_norm(k, _w(W, pre + ".k.norm"), eps).view(T, G, D)
    o = distance_attention(q, k, v.view(T, G, Dv), m["scale"], m.get("softcap"), (m.get("mask") or {}).get("size"))
    return o.reshape(T, H * Dv) @ _w(W, pre + ".o").T + _w(W, pre + ".o.b")


# ------------------------------------------------------------- recurrence
def short_conv(u, w, b):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_{t - taps + 1 + j} + b, zeros before the start."""
    T, C = u.shape
    taps = w.shape[1]
    pad = torch.cat([torch.zeros((taps - 1, C), dtype=F64), u])
    y = torch.zeros_like(u) + b
    for j in range(taps):
        y = y + pad[j:j + T] * w[:, j][None, :]
    return y


def selective_recurrence(x, B, C, dt, a_log, d_skip):
    """S_t = exp(-exp(a_log_h) dt_t) S_{t-1} + dt_t B_t x_t^T, y_t = S_t^T C_t + d_h x_t; x [T, H, P], B and C
    [T, G, N] (head h reads group h // (H/G)), dt [T, H]."""
    T, H, P = x.shape
    rep = H // B.shape[1]
    Bh, Ch = B.repeat_interleave(rep, dim=1), C.repeat_interleave(rep, dim=1)
    S = torch.zeros((H, B.shape[2], P), dtype=F64)
    rate = torch.exp(a_log)
    out = []
    for t in range(T):
        S = torch.exp(-rate * dt[t])[:, None, None] * S + (dt[t][:, None] * Bh[t])[:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hnp,hn->hp", S, Ch[t]) + d_skip[:, None] * x[t])
    return torch.stack(out)


def gated_group_norm(y, z, w, groups: int, eps: float):
    """y silu(z), then an RMS norm of each of ``groups`` equal parts, times w."""
    T, n = y.shape
    g = (y * silu(z)).view(T, groups, n // groups)
    return rms_norm(g, None, eps).reshape(T, n) * w


def state_space_mixer(h, m: dict, W, pre: str, eps: float):
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    row = h @ _w(W, pre + ".in").T
    z, xbc, dt = row[:, :inner], row[:, inner:2 * inner + 2 * G * N], row[:, 2 * inner + 2 * G * N:]
    u = silu(short_conv(xbc, _w(W, pre + ".conv"), _w(W, pre + ".conv.b")))
    x, B, C = u[:, :inner].view(T, H, P), u[:, inner:inner + G * N].view(T, G, N), u[:, inner + G * N:].view(T, G, N)
    dt = torch.nn.functional.softplus(dt + _w(W, pre + ".dt_bias"), threshold=1e9)
    y = selective_recurrence(x, B, C, dt, _w(W, pre + ".A_log"), _w(W, pre + ".D")).reshape(T, inner)
    return gated_group_norm(y, z, _w(W, pre + ".norm"), m["norm_groups"], eps) @ _w(W, pre + ".o").T


def parallel_mixer(h, m: dict, W, pre: str, eps: float):
    return (m["left_scale"] * attention_mixer(h, m["left"], W, pre + ".left", eps)
            + m["right_scale"] * state_space_mixer(h, m["right"], W, pre + ".right", eps))


# ----------------------------------------------------------- feed-forward
def clamped_unit(g, u, limit: float):
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def dense(h, W, pre: str, limit: float):
    return clamped_unit(h @ _w(W, pre + ".gate").T, h @ _w(W, pre + ".up").T, limit) @ _w(W, pre + ".down").T


def route(z, top: int):
    """(chosen experts [T, top], their weights): the ``top`` largest sigmoids, not renormalized; ties: the
    lower index."""
    s = torch.sigmoid(z)
    ids = torch.sort(s, dim=-1, descending=True, stable=True).indices[:, :top]
    return ids, torch.gather(s, 1, ids)


def experts(h, mlp: dict, W, pre: str):
    """sum over a token's experts of expert(weight * h): the weight enters before the expert."""
    ids, weights = route(h @ _w(W, pre + ".router").T, mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(ids[t].tolist(), weights[t]):
            out[t] += dense((w * h[t])[None], W, f"{pre}.e{e}", mlp["expert"]["limit"])[0]
    return out


def feed_forward(h, mlp: dict, W, pre: str):
    return dense(h, W, pre, mlp["limit"]) if mlp["kind"] == "dense" else experts(h, mlp, W, pre)


# ------------------------------------------------------------------ model
def forward(cfg: dict, W: Dict[str, torch.Tensor], ids: List[int], streams: Optional[list] = None):
    """Logits [T, vocab] float64 of one sequence; ``streams`` (a list) receives the stream after
    every layer."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = _w(W, "embed")[torch.tensor(ids)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}"
        y = parallel_mixer(rms_norm(x, _w(W, p + ".norm1"), eps), layer["mixer"], W, p + ".mix", eps)
        x = x + m * rms_norm(y, _w(W, p + ".norm1b"), eps)
        if layer.get("mlp"):
            y = feed_forward(rms_norm(x, _w(W, p + ".norm2"), eps), layer["mlp"], W, p + ".mlp")
            x = x + m * rms_norm(y, _w(W, p + ".norm2b"), eps)
        if streams is not None:
            streams.append(x.clone())
    return rms_norm(x, _w(W, "final.norm"), eps) @ _w(W, "embed").T


# ----------------------------------------------------------- model folders
_DT = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32, "I64": torch.int64}


def read_safetensors(path: str) -> Dict[str, torch.Tensor]:
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, e in header.items():
        if name == "__metadata__":
            continue
        lo, hi = e["data_offsets"]
        out[name] = torch.frombuffer(bytearray(data[lo:hi]), dtype=_DT[e["dtype"]]).reshape(e["shape"]).clone()
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
