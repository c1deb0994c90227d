"""Small Dimudra configurations (sizes unlike any real model's, several values of every option), a writer of random model
folders for them, and the plain implementation's logits."""
from __future__ import annotations

import copy
import json
import os

import torch

from logssms_b200.config import make_model_config
from logssms_b200.weights import write_random_model

from plain import dimudra_plain as P


def _left(heads, kv_heads, dim, vdim, window, scale):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    return m


def _right(inner, state, dt_rank, conv):
    return {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}


def _parallel(left, right, left_scale=1.0, right_scale=1.0):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}}


def _hgrn2(heads, dim, vdim):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}}


def _attention(heads, kv_heads, dim, vdim, scale, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "attention", "mixer": m}


def _moe(experts, top, count, keep, ff, shared):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}},
            "shared": {"ff": shared}}


def _model(width, vocab, eps, scale, taps, loop, layers):
    return {"architecture": "Dimudra", "layers": layers, "norm": {"eps": eps}, "embedding": {"scale": scale}, "canon": {"taps": taps},
            "loop": dict(zip(("start", "stop", "times"), loop)), "vocab": vocab, "width": width}


# A: all three mixers; a window (20) shorter than a page of 64 and crossed many times; grouped queries 3 to 1; value heads of
# another size than key heads; a rotation over part of the head; a loop over two layers, three passes; a layer without
# feed-forward
DIMU_A = _model(64, 211, 1e-5, 3.0, 3, (1, 3, 3), [
    {**_parallel(_left(6, 2, 16, 24, 20, 0.3), _right(72, 12, 5, 4), 0.8, 1.3), "mlp": _moe(12, 3, 4, 2, 16, 24)},
    {**_hgrn2(3, 16, 24), "mlp": _moe(6, 2, 3, 2, 24, 8)},
    {**_attention(4, 2, 16, 8, 0.35, (8, 500.0)), "mlp": _moe(8, 4, 2, 1, 16, 32)},
    {**_parallel(_left(2, 1, 32, 16, 33, 0.2), _right(40, 16, 8, 2), 1.5, 0.6), "mlp": None},
])

# B: rotary attention first, the whole head rotated; a window (70) just past a page; one tap of the input convolution; the
# whole model looped twice
DIMU_B = _model(96, 333, 1e-6, 0.5, 1, (0, 3, 2), [
    {**_attention(4, 4, 32, 32, 0.25, (32, 10000.0)), "mlp": _moe(4, 1, 1, 1, 40, 16)},
    {**_hgrn2(2, 32, 40), "mlp": None},
    {**_parallel(_left(4, 1, 32, 32, 70, 0.25), _right(64, 36, 3, 3), 1.0, 1.0), "mlp": _moe(16, 5, 8, 4, 8, 40)},
])

# C: sizes of 1 where the design allows them: one head, one state per channel, a step rank of 1, a window of 1, one expert, one
# tap in the scan's convolution; a loop of one pass
DIMU_C = _model(48, 130, 1e-5, 1.0, 2, (0, 2, 1), [
    {**_parallel(_left(1, 1, 2, 1, 1, 0.5), _right(8, 1, 1, 1), 1.0, 2.0), "mlp": _moe(1, 1, 1, 1, 8, 1)},
    {**_hgrn2(1, 1, 2), "mlp": _moe(2, 1, 2, 1, 4, 4)},
    {**_attention(1, 1, 2, 1, 0.7, (2, 100.0)), "mlp": None},
])

# D: recurrent layers only (no paged cache at all); an empty loop
DIMU_D = _model(40, 90, 1e-5, 5.0, 5, (1, 1, 4), [
    {**_hgrn2(2, 48, 72), "mlp": _moe(9, 4, 3, 2, 24, 16)},
    {**_hgrn2(4, 8, 16), "mlp": None},
])

# E: nothing is a multiple of 8; windows of 64 (a page) and 400 (never reached); no rotation; a loop of a single layer
DIMU_E = _model(54, 177, 1e-5, 1.7, 4, (2, 3, 4), [
    {**_parallel(_left(4, 2, 10, 6, 64, 0.35), _right(50, 5, 7, 5), -0.7, 1.1), "mlp": _moe(10, 3, 5, 3, 22, 14)},
    {**_attention(3, 1, 22, 18, 0.3), "mlp": _moe(6, 6, 2, 2, 10, 6)},
    {**_hgrn2(3, 20, 5), "mlp": _moe(14, 2, 2, 1, 18, 9)},
    {**_parallel(_left(2, 2, 16, 16, 400, 0.3), _right(33, 70, 2, 4), 1.0, 0.4), "mlp": _moe(7, 2, 1, 1, 12, 30)},
])


def random_dimudra(seed: int) -> dict:
    """A configuration with every size and option drawn at random within what config.json allows."""
    import random
    rng = random.Random(seed)
    n = rng.randint(2, 5)
    layers = []
    for _ in range(n):
        kv, dim = rng.choice([1, 2, 3]), rng.choice([8, 16, 24, 32, 64])
        heads, vdim = kv * rng.choice([1, 2, 4]), rng.choice([4, 8, 16, 24, 40])
        r = rng.random()
        if r < 0.4:
            mixer = _parallel(_left(heads, kv, dim, vdim, rng.choice([1, 3, 17, 64, 65, 100, 300]), rng.choice([0.1, 0.3])),
                              _right(8 * rng.randint(1, 12) + rng.choice([0, 0, 3]), rng.choice([1, 4, 7, 16, 24, 64, 130]), rng.randint(1, 12),
                                     rng.randint(1, 6)), rng.choice([0.5, 1.0, 1.4]), rng.choice([0.6, 1.0]))
        elif r < 0.7:
            mixer = _hgrn2(rng.randint(1, 4), rng.choice([4, 8, 16, 32, 80]), vdim)
        else:
            mixer = _attention(heads, kv, dim, vdim, rng.choice([0.1, 0.3]), None if rng.random() < 0.2 else (2 * rng.randint(1, dim // 2), 3000.0))
        count = rng.choice([1, 2, 4])
        per = rng.randint(1, 4)
        keep = rng.randint(1, count)
        top = rng.randint(1, min(keep * per, 5))
        layers.append({**mixer, "mlp": None if rng.random() < 0.2 else _moe(count * per, top, count, keep, rng.randint(3, 40), rng.randint(3, 40))})
    start = rng.randint(0, n - 1)
    loop = (start, rng.randint(start + 1, n), rng.randint(1, 3))
    return _model(8 * rng.randint(4, 12), rng.randint(60, 400), rng.choice([1e-5, 1e-6]), rng.choice([0.5, 1.0, 12.0]), rng.randint(1, 6), loop, layers)


DIMU = {"A": DIMU_A, "B": DIMU_B, "C": DIMU_C, "D": DIMU_D, "E": DIMU_E}
DIMU.update({f"R{seed}": random_dimudra(seed) for seed in range(1, 9)})


def calm_routers(tensors: dict) -> None:
    """Make the routers' choices follow their corrections: no close calls, which rounding of their input would turn."""
    for name, t in tensors.items():
        if name.endswith("router"):
            tensors[name] = (t.float() * 0.002).to(t.dtype)
        elif name.endswith("correction"):
            tensors[name] = (t.float() * 6.0).to(t.dtype)


def make_dimudra_dir(path, raw: dict, seed: int = 0, dtype=torch.float32, sharp: float = 1.0, calm: bool = False) -> str:
    """Random weights for `raw` in `path`.  `sharp` scales the attentions' scores (their `scale`) so that the softmax picks
    single keys: a missing or surplus key, or the added one that is left out, then moves the logits far beyond any tolerance.
    `calm`: see `calm_routers`."""
    from safetensors.torch import load_file, save_file
    raw = copy.deepcopy(raw)
    for layer in raw["layers"]:
        if layer["type"] == "parallel":
            layer["mixer"]["left"]["scale"] *= sharp
        elif layer["type"] == "attention":
            layer["mixer"]["scale"] *= sharp
    out = write_random_model(make_model_config(raw), str(path), seed=seed, dtype=dtype, perturb=True)
    if calm:
        file = os.path.join(out, "model.safetensors")
        tensors = load_file(file)
        calm_routers(tensors)
        save_file(tensors, file)
    return out


def read_folder(model_dir: str):
    from safetensors.torch import load_file
    with open(os.path.join(model_dir, "config.json")) as f:
        config = json.load(f)
    return config, load_file(os.path.join(model_dir, "model.safetensors"))


def plain_logits(model_dir: str, ids, dtype=torch.float64) -> torch.Tensor:
    """The plain model's logits at every position, from the folder's stored weights (in `dtype` throughout)."""
    config, tensors = read_folder(model_dir)
    return P.forward(config, tensors, list(ids), dtype=dtype).double()


def row_errors(got: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
    """Per position: root mean square of the logits' difference (its mean over the vocabulary taken off) over the root
    mean square of the wanted logits."""
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape, (got.shape, want.shape)
    assert torch.isfinite(got).all(), "engine produced non-finite logits"
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt().clamp_min(1e-30)


TOL = {"float32": 3e-4, "bfloat16": 5e-2}
