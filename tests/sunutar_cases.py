"""Tiny Sunutar configurations for the tests.  Their layers differ in every size, constant and order and include
the values a model could happen to make equal or 1: one kv head, as many kv heads as heads, keys larger and
smaller than values, windows of 1, 5, 33, 70, one beyond every request and none, no soft cap, one group and as
many groups as heads, one head, one norm part and several (also parts that cut heads), one tap, two and five,
one expert of each token, all of them and one expert alone, layers without feed-forward, factors of 1 and
others, and sizes that fit no 16-byte access."""

from __future__ import annotations


def left(heads, kv, dim, vdim, scale, window=None, cap=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    if cap is not None:
        m["softcap"] = cap
    return m


def right(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff, limit):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def layer(lm, rm, ls, rs, mlp):
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": lm, "right": rm, "left_scale": ls, "right_scale": rs}}


A = {"architecture": "Sunutar", "vocab": 211, "width": 48, "norm": {"eps": 1e-6}, "residual_mult": 0.55,
     "layers": [layer(left(4, 2, 16, 8, 0.4, 5, 6.0), right(3, 16, 8, 1, 3, 4), 0.6, 1.1, moe(5, 2, 24, 1.5)),
                layer(left(6, 1, 8, 24, 0.5, 33, 20.0), right(4, 8, 24, 2, 2, 1), 1.3, 0.7, None),
                layer(left(2, 2, 24, 16, 0.3, None, 9.0), right(2, 12, 16, 2, 4, 3), 1.0, 0.4, dense(40, 0.9))]}
# sizes that no 16-byte access fits; a window of one token; one tap; norm parts that cut heads
B = {"architecture": "Sunutar", "vocab": 97, "width": 50, "norm": {"eps": 1e-5}, "residual_mult": 1.0,
     "layers": [layer(left(3, 3, 10, 6, 0.5, 1, 4.0), right(3, 7, 9, 3, 1, 7), 1.0, 1.0, dense(22, 3.0)),
                layer(left(3, 1, 6, 10, 0.6, 70, 12.0), right(1, 9, 11, 1, 5, 1), 0.9, 1.2, moe(3, 3, 14, 0.7)),
                layer(left(5, 5, 14, 6, 0.4, 9), right(5, 6, 3, 5, 3, 2), 0.5, 0.8, moe(1, 1, 10, 2.0))]}
# sizes in multiples of 64: the tensor-core attention of every kind
C = {"architecture": "Sunutar", "vocab": 150, "width": 128, "norm": {"eps": 1e-5}, "residual_mult": 0.8,
     "layers": [layer(left(4, 1, 64, 64, 0.2, 70, 15.0), right(4, 64, 64, 1, 4, 2), 0.7, 0.6, dense(128, 1.2)),
                layer(left(2, 2, 64, 128, 0.25, None, 25.0), right(2, 64, 128, 2, 4, 1), 1.2, 0.9, moe(6, 1, 64, 1.0)),
                layer(left(8, 2, 128, 64, 0.15, 33, 10.0), right(6, 32, 64, 3, 2, 6), 0.8, 1.4, moe(4, 2, 32, 2.5))]}
# sizes in multiples of 16 but not of 64, a state beyond 128, a window beyond every request
D = {"architecture": "Sunutar", "vocab": 320, "width": 160, "norm": {"eps": 1e-6}, "residual_mult": 0.9,
     "layers": [layer(left(6, 3, 48, 32, 0.2, 1000, 18.0), right(5, 24, 48, 5, 5, 4), 0.5, 1.5, moe(9, 3, 48, 1.0)),
                layer(left(6, 2, 32, 80, 0.3, 40, 7.0), right(2, 80, 144, 1, 3, 5), 1.1, 0.3, dense(80, 1.7))]}
CASES = {"A": (A, 5, 8), "B": (B, 9, 4), "C": (C, 13, 16), "D": (D, 17, 32)}   # config, seed, page size
# peaked scores, gates on both sides of their limits, step sizes and decays from a token to hundreds: leaving a
# step out moves the logits
STD_OF = {"embed": 0.6, ".router": 0.6, ".mlp": 0.2, ".conv.b": 0.3, ".conv": 0.5, ".dt_bias": 2.5, ".A_log": 1.5,
          ".right.D": 1.0, ".q.b": 0.5, ".k.b": 0.5, ".v.b": 0.5, ".o.b": 0.5, ".q": 0.3, ".k": 0.3, ".right.in": 0.25}


def make_model(folder: str, cfg: dict, seed: int) -> str:
    """The weights are stored in bfloat16, as a served model's are."""
    import torch
    from servelab_b200.config import config_from_dict
    from servelab_b200.weights import write_random_model
    return write_random_model(folder, config_from_dict(cfg), seed, dtype=torch.bfloat16, std=0.15, norm_std=0.3,
                              std_of=STD_OF)
