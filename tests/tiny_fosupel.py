"""Small Fosupel configurations (sizes unlike any real model's, several values of every option), a writer of random model
folders for them, and the plain implementation's logits."""
from __future__ import annotations

import copy

import torch

from logssms_b200.config import make_model_config
from logssms_b200.weights import write_random_model

from plain import fosupel_plain as P
from tiny_dimudra import TOL, read_folder, row_errors  # noqa: F401  (used by the tests of this design)


def rotation(dims, base, factor=None):
    rot = {"dims": dims, "base": base}
    if factor is not None:
        rot["scaling"] = {"factor": factor}
    return rot


def left(heads, kv_heads, dim, vdim, window, keep, scale, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window, "keep_first": keep}
    if rot is not None:
        m["rot"] = rotation(*rot)
    return m


def right(heads, dim, vdim, rot=None, decay=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [1.0 - 2.0 ** -(2 + 3 * h) for h in range(heads)]}
    if rot is not None:
        m["rot"] = rotation(*rot)
    return m


def parallel(a, b, left_scale=1.0, right_scale=1.0):
    return {"type": "parallel", "mixer": {"left": a, "right": b, "left_scale": left_scale, "right_scale": right_scale}}


def latent(heads, dim, rot_dim, vdim, rank, scale, base=1000.0):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
                                                  "rot": None if rot_dim == 0 else rotation(rot_dim, base)}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": None if shared is None else {"ff": shared}}


def model(width, vocab, eps, mult, cap, loop, layers):
    raw = {"architecture": "Fosupel", "layers": layers, "norm": {"eps": eps}, "residual_mult": mult, "logit_softcap": cap, "vocab": vocab,
           "width": width}
    if loop is not None:
        raw["loop"] = dict(zip(("start", "stop", "times"), loop))
    return raw


# A: both mixers, both feed-forwards and none; a window (20) shorter than a page of 64 and crossed many times, kept tokens (5) within
# a page; grouped queries 3 to 1; value heads of another size than key heads; rotations over part of a head, with a factor and
# without; a loop of three passes that opens behind the first layer
FOSU_A = model(64, 211, 1e-5, 0.6, 12.0, (1, 3, 3), [
    {**parallel(left(6, 2, 16, 24, 20, 5, 0.3, (8, 500.0, 3.0)), right(3, 16, 24, (8, 40.0)), 0.8, 1.3), "mlp": dense(72)},
    {**latent(4, 16, 8, 24, 40, 0.25), "mlp": moe(6, 2, 24, 8)},
    {**parallel(left(4, 4, 32, 16, 33, 70, 0.2, (32, 1e4)), right(2, 32, 8, (32, 1e4, 2.0)), 1.5, 0.6), "mlp": moe(8, 3, 16, 32)},
    {**latent(3, 24, 16, 16, 32, 0.2), "mlp": None},
])

# B: the whole model looped twice (the first layer opens a pass); latent attention first; a window (70) just past a page, no kept
# tokens; one key/value head; no shared expert
FOSU_B = model(96, 333, 1e-6, 1.0, 30.0, (0, 2, 2), [
    {**latent(8, 32, 16, 32, 64, 0.2), "mlp": moe(4, 1, 40, None)},
    {**parallel(left(4, 1, 32, 32, 70, 0, 0.25, (20, 3000.0, 1.5)), right(4, 32, 40, (10, 90.0)), 1.0, 1.0), "mlp": dense(130)},
])

# C: sizes of 1 where the design allows them: one head, a window of 1, one kept token, one expert, a decay of 1 (nothing is
# forgotten); no rotation; a latent attention without a rotated part; a loop of one pass
FOSU_C = model(48, 130, 1e-5, 1.4, 5.0, (0, 1, 1), [
    {**parallel(left(1, 1, 2, 1, 1, 1, 0.5), right(1, 1, 1, None, [1.0]), 1.0, 2.0), "mlp": moe(1, 1, 8, 1)},
    {**latent(1, 2, 0, 1, 1, 0.7), "mlp": dense(1)},
    {**parallel(left(2, 2, 2, 2, 3, 2, 0.5, (2, 10.0, 5.0)), right(2, 2, 3, (2, 10.0), [0.5, 1.0]), 0.5, 1.0), "mlp": None},
])

# D: no latent attention, no loop, no window at all in one layer; many heads to one key/value head (more than a tile of 16)
FOSU_D = model(40, 90, 1e-5, 0.8, 20.0, None, [
    {**parallel(left(18, 1, 16, 8, None, 0, 0.3, (16, 300.0)), right(2, 48, 72, (48, 1e5)), 0.7, 0.9), "mlp": dense(24)},
    {**parallel(left(20, 4, 16, 8, 64, 64, 0.3, (4, 7.0, 9.0)), right(4, 8, 16), 1.0, -0.5), "mlp": moe(9, 4, 24, 16)},
])

# E: nothing is a multiple of 8; windows of 64 (a page) and 400 (never reached), kept tokens past a page; a loop of a single layer
FOSU_E = model(54, 177, 1e-5, 0.5, 9.0, (2, 3, 4), [
    {**parallel(left(4, 2, 10, 6, 64, 67, 0.35, (6, 50.0, 2.5)), right(3, 20, 5, (6, 50.0)), -0.7, 1.1), "mlp": moe(10, 3, 22, 14)},
    {**latent(3, 10, 6, 7, 20, 0.3), "mlp": dense(37)},
    {**parallel(left(3, 3, 7, 9, 31, 3, 0.3), right(1, 33, 12, (10, 9.0)), 1.0, 0.4), "mlp": moe(7, 2, 12, 30)},
    {**parallel(left(5, 5, 22, 18, 400, 9, 0.3, (22, 1e6, 1.1)), right(2, 6, 6), 1.0, 0.4), "mlp": None},
])


def random_fosupel(seed: int) -> dict:
    """A configuration with every size and option drawn at random within what config.json allows."""
    import random
    rng = random.Random(seed)
    n = rng.randint(2, 5)
    rot_of = lambda dim: None if rng.random() < 0.2 or dim < 2 else (2 * rng.randint(1, dim // 2), rng.choice([30.0, 1e4, 1e6])) + \
        ((rng.choice([1.5, 8.0]),) if rng.random() < 0.5 else ())
    layers = []
    for _ in range(n):
        kv, dim = rng.choice([1, 2, 3, 4]), rng.choice([8, 16, 32, 48, 64])
        heads, vdim = kv * rng.choice([1, 2, 4]), rng.choice([4, 8, 16, 24, 64])
        if rng.random() < 0.6:
            dk, hr = rng.choice([4, 16, 32, 80]), rng.randint(1, 4)
            mixer = parallel(left(heads, kv, dim, vdim, rng.choice([1, 3, 17, 64, 65, 100]), rng.choice([0, 1, 16, 63, 64, 80]), rng.choice([0.1, 0.3]),
                                  rot_of(dim)),
                             right(hr, dk, vdim, rot_of(dk), [rng.choice([0.3, 0.9, 0.984, 0.9995, 1.0]) for _ in range(hr)]),
                             rng.choice([0.5, 1.0, 1.4]), rng.choice([0.6, 1.0]))
        else:
            mixer = latent(heads, dim, rng.choice([2, 8, 16, 32]), vdim, rng.choice([16, 32, 56, 64]), rng.choice([0.1, 0.25]))
        ff = rng.random()
        experts = rng.randint(1, 12)
        layers.append({**mixer, "mlp": None if ff < 0.15 else dense(rng.randint(3, 90)) if ff < 0.5 else
                       moe(experts, rng.randint(1, experts), rng.randint(3, 40), None if rng.random() < 0.2 else rng.randint(3, 40))})
    start = rng.randint(0, n - 1)
    return model(8 * rng.randint(4, 12), rng.randint(60, 400), rng.choice([1e-5, 1e-6]), rng.choice([0.4, 1.0]), rng.choice([6.0, 40.0]),
                 (start, rng.randint(start + 1, n), rng.randint(1, 3)), layers)


FOSU = {"A": FOSU_A, "B": FOSU_B, "C": FOSU_C, "D": FOSU_D, "E": FOSU_E}
FOSU.update({f"R{seed}": random_fosupel(seed) for seed in range(1, 9)})


def make_fosupel_dir(path, raw: dict, seed: int = 0, dtype=torch.float32, sharp: float = 1.0, calm: bool = False) -> str:
    """Random weights for `raw` in `path`.  `sharp` scales the attentions' scores (their `scale`) so that the softmax picks
    single keys: a missing or surplus key then moves the logits far beyond any tolerance.  `calm`: every router chooses all of its
    experts, so that rounding turns no close call."""
    raw = copy.deepcopy(raw)
    for layer in raw["layers"]:
        m = layer["mixer"]["left"] if layer["type"] == "parallel" else layer["mixer"]
        m["scale"] *= sharp
        if calm and layer["mlp"] is not None and layer["mlp"]["kind"] == "moe":
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return write_random_model(make_model_config(raw), str(path), seed=seed, dtype=dtype, perturb=True)


def plain_logits(model_dir: str, ids, dtype=torch.float64) -> torch.Tensor:
    """The plain model's logits at every position, from the folder's stored weights (in `dtype` throughout)."""
    config, tensors = read_folder(model_dir)
    return P.forward(config, tensors, list(ids), dtype=dtype).double()
