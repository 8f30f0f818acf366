"""Tiny Vufadra configurations for the tests.  Their layers differ in every size, constant and order
and include the values a model could happen to make equal or 1: one head, one kv head, as many kv
heads as heads, keys larger and smaller than values, a rotation of part of a head, of all of it and
none, interpolated and plain frequencies, chunks of 1, 5, 33, 70 and one beyond every request, no
mask, one tap, two taps and five, one diagonal block and several, no loop, a loop over one layer, over
all layers and a single pass, no bigram embedding and one with few buckets, layers without
feed-forward, every mixer as the first layer, and sizes that fit no 16-byte access."""

from __future__ import annotations

import json
import os


def delta(heads, dim, rank):
    return "general_delta", {"heads": heads, "dim": dim, "rank": rank}


def rglru(width, blocks, taps):
    return "rglru", {"width": width, "blocks": blocks, "conv": taps}


def parallel(left, right):
    """left: (heads, kv, dim, vdim, scale, chunk, rot); right: (heads, dim, rank)."""
    heads, kv, dim, vdim, scale, chunk, rot = left
    lm = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk is not None:
        lm["mask"] = {"size": chunk}
    if rot:
        lm["rot"] = {"base": rot[0], "dims": rot[1]}
        if len(rot) > 2:
            lm["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[2]))
    rh, rd, rank = right
    return "parallel", {"left": lm, "right": {"heads": rh, "dim": rd, "rank": rank}}


def layer(mixer, ff):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def bigram(buckets, mul_prev, mul_cur):
    return {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}


# the parallel layer first; the two middle layers run three times
A = {"architecture": "Vufadra", "vocab": 211, "width": 48, "norm": {"eps": 1e-6}, "embedding": bigram(101, 31, 7),
     "loop": {"start": 1, "stop": 3, "times": 3},
     "layers": [layer(parallel((4, 2, 16, 8, 0.25, 5, (500.0, 8, (4.0, 64, 8.0, 1.0))), (3, 8, 6)), 40),
                layer(rglru(36, 3, 3), 24),
                layer(delta(3, 8, 5), None),
                layer(parallel((2, 1, 8, 24, 0.35, 33, (10000.0, 8)), (2, 12, 4)), 32)]}
# no loop, no bigram embedding, sizes that no 16-byte access fits; a chunk of one token; one tap
B = {"architecture": "Vufadra", "vocab": 97, "width": 50, "norm": {"eps": 1e-5},
     "layers": [layer(delta(1, 14, 3), 22),
                layer(parallel((3, 3, 10, 6, 0.3, 1, None), (1, 6, 3)), 14),
                layer(rglru(30, 5, 1), None),
                layer(parallel((3, 1, 6, 10, 0.4, None, (50.0, 4)), (3, 10, 7)), 18),
                layer(delta(5, 6, 2), 10)]}
# sizes in multiples of 64 (the tensor-core attention of every kind), the whole model twice
C = {"architecture": "Vufadra", "vocab": 150, "width": 128, "norm": {"eps": 1e-5}, "embedding": bigram(3, 1, 1),
     "loop": {"start": 0, "stop": 3, "times": 2},
     "layers": [layer(rglru(128, 1, 5), 64),
                layer(parallel((4, 1, 64, 64, 0.06, 70, (1e6, 32, (2.0, 128, 32.0, 1.0))), (2, 64, 16)), 96),
                layer(delta(2, 64, 16), 64)]}
# sizes in multiples of 16 but not of 64, heads beyond 128, a loop of a single pass over one layer
D = {"architecture": "Vufadra", "vocab": 320, "width": 160, "norm": {"eps": 1e-6}, "embedding": bigram(640, 127, 8191),
     "loop": {"start": 2, "stop": 3, "times": 1},
     "layers": [layer(delta(2, 136, 24), 80),
                layer(rglru(96, 6, 2), 64),
                layer(parallel((6, 3, 48, 32, 0.14, 1000, (2e5, 16)), (4, 32, 8)), 48),
                layer(parallel((6, 2, 32, 80, 0.15, 40, (3e4, 32, (8.0, 32, 4.0, 0.5))), (1, 48, 8)), None)]}
CASES = {"A": (A, 5, 8), "B": (B, 9, 4), "C": (C, 13, 16), "D": (D, 17, 32)}   # config, seed, page size
# scores of sigmoid attention spread over both sides of zero; decays, rates, mixes, shifts and taps large
# enough that leaving one out moves the logits
STD_OF = {"embed": 0.6, "bigram": 0.6, "loop.in": 0.08, "loop.step": 0.4, ".shift": 0.5, ".mu.": 0.5, ".pb": 1.5,
          ".mlp": 0.15, ".conv.b": 0.3, ".conv": 0.5, ".w0": 1.5, ".w1": 0.3, ".w2": 0.6, ".a.b": 1.0, ".right.u": 1.0,
          ".lam": 2.0, ".ra": 0.4, ".ri": 0.4, ".q": 0.3, ".k": 0.3}


def make_model(folder: str, cfg: dict, seed: int, drop_rank: bool = False) -> str:
    """The weights are stored in bfloat16, as a served model's are.  ``drop_rank``: config.json is
    written without the bottleneck sizes of the decays, which the loader then reads from the tensors."""
    import torch
    from servelab_b200.config import config_from_dict
    from servelab_b200.weights import write_random_model
    write_random_model(folder, config_from_dict(cfg), seed, dtype=torch.bfloat16, std=0.15, norm_std=0.3,
                       std_of=STD_OF)
    if drop_rank:
        path = os.path.join(folder, "config.json")
        with open(path) as f:
            written = json.load(f)
        for entry in written["layers"]:
            for m in (entry["mixer"], entry["mixer"].get("right", {})):
                m.pop("rank", None)
        with open(path, "w") as f:
            json.dump(written, f, indent=1)
    return folder
