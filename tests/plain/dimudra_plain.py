"""A plain, slow Dimudra: one function per mechanism, written from the design's equations in float64 tensor operations,
token by token where the design is a recurrence.  It shares no code with the engine; the engine's tests compare against it.

A model is (config mapping, {tensor name: tensor}); a request is a list of token ids.  `forward` returns the logits at
every position and, on request, the stream after every layer run.  With another `dtype` than float64 every tensor and every
intermediate result is of that dtype (angles excepted): what rounding alone does to a model.
"""
from __future__ import annotations

import torch

F = torch.float64
silu = torch.nn.functional.silu


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def short_conv(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the sequence's start."""
    T, taps = u.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u], 0)
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + padded[j:j + T] * w[:, j]
    return y


def input_conv(h, w):
    """What a mixer reads: the normed rows plus their causal convolution over time."""
    return h + short_conv(h, w)


def rotate_halves(x, positions, rot):
    """x [T, heads, d]: of every head's first rot.dims columns, column i and column i + dims/2 turn by position * base^(-2i/dims)
    (`rot` None: nothing turns)."""
    if rot is None:
        return x
    dims, base = int(rot["dims"]), float(rot["base"])
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=F)
    a = positions.to(F)[:, None] * f[None, :]
    cos, sin = torch.cos(a)[:, None, :].to(x.dtype), torch.sin(a)[:, None, :].to(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], -1)


def softmax_attention(q, k, v, scale, window, extra):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; query head h reads key/value head h // (H / G); position i sees j with
    0 <= i - j < window (None: every j <= i); the denominator also holds `extra` times exp(0)."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i if window is None else (j <= i) & (i - j < window)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(~seen[None], float("-inf"))
    m = s.amax(-1, keepdim=True).clamp_min(0.0)
    e = torch.exp(s - m)
    p = e / (e.sum(-1, keepdim=True) + extra * torch.exp(-m))
    return torch.einsum("hij,jhd->ihd", p, v)


def window_attention(h, p, m, eps):
    """The left branch of a 'parallel' mixer: biases in the projections, q and k normed over their whole rows, no rotation, a
    window, an ordinary softmax, an output gate per element."""
    T, H, G, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = (rms(h @ p["q"].T + p["q.b"], eps) * p["q.norm"]).view(T, H, d)
    k = (rms(h @ p["k"].T + p["k.b"], eps) * p["k.norm"]).view(T, G, d)
    v = (h @ p["v"].T + p["v.b"]).view(T, G, dv)
    window = None if m.get("mask") is None else int(m["mask"]["size"])
    o = softmax_attention(q, k, v, float(m["scale"]), window, 0.0).reshape(T, H * dv)
    return (o * torch.sigmoid(h @ p["g"].T)) @ p["o"].T


def rotary_attention(h, p, m, eps):
    """The 'attention' mixer: q and k rotated, then divided by their root mean square per head; one added to the softmax's
    denominator; an output gate per element."""
    T, H, G, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(T)
    q = rms(rotate_halves((h @ p["q"].T).view(T, H, d), pos, m.get("rot")), eps)
    k = rms(rotate_halves((h @ p["k"].T).view(T, G, d), pos, m.get("rot")), eps)
    v = (h @ p["v"].T).view(T, G, dv)
    o = softmax_attention(q, k, v, float(m["scale"]), None, 1.0).reshape(T, H * dv)
    return (o * torch.sigmoid(h @ p["g"].T)) @ p["o"].T


def selective_scan(x, dt, A, B, C, D):
    """x, dt [T, inner], A [inner, state], B, C [T, state]: S <- exp(dt A) S + dt x B, y = S C + D x, from S = 0."""
    S = torch.zeros_like(A)
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y


def mamba(h, p, m):
    """The right branch of a 'parallel' mixer."""
    inner, rank, n = int(m["inner"]), int(m["dt_rank"]), int(m["state"])
    xz = h @ p["in"].T
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(short_conv(x, p["conv"]) + p["conv.b"])
    low = x @ p["x"].T
    dt = torch.nn.functional.softplus(low[:, :rank] @ p["dt"].T + p["dt.b"])
    y = selective_scan(x, dt, -torch.exp(p["A_log"]), low[:, rank:rank + n], low[:, rank + n:], p["D"])
    return (y * silu(z)) @ p["o"].T


def gated_recurrence(q, f, v):
    """q, f [T, H, d], v [T, H, dv]: S <- diag(f) S + (1 - f) v^T, o = S^T q, from S = 0."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    o = torch.zeros_like(v)
    for t in range(T):
        S = f[t][:, :, None] * S + (1 - f[t])[:, :, None] * v[t][:, None, :]
        o[t] = (q[t][:, :, None] * S).sum(1)
    return o


def hgrn2(h, p, m, eps):
    T, H, d, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = silu(h @ p["q"].T).view(T, H, d)
    f = (p["lower"] + (1 - p["lower"]) * torch.sigmoid(h @ p["f"].T + p["f.b"])).view(T, H, d)
    v = (h @ p["v"].T).view(T, H, dv)
    o = rms(gated_recurrence(q, f, v), eps) * p["norm"]
    return o.reshape(T, H * dv) @ p["o"].T


def gated_ff(h, p):
    return (silu(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def route(z, correction, top, groups, keep):
    """Router outputs z [T, n] -> weights [T, n] (0: not chosen), token by token."""
    s = torch.sigmoid(z)
    weights = torch.zeros_like(s)
    n = z.shape[1]
    per = n // groups
    for t in range(z.shape[0]):
        choice = [float(c) for c in (s[t] + correction)]
        score = [sum(sorted(choice[g * per:(g + 1) * per], reverse=True)[:2]) for g in range(groups)]
        kept = sorted(range(groups), key=lambda g: -score[g])[:keep]
        allowed = [e for e in range(n) if e // per in kept]
        chosen = sorted(allowed, key=lambda e: -choice[e])[:top]
        total = sum(s[t, e] for e in chosen) + 1e-20
        for e in chosen:
            weights[t, e] = s[t, e] / total
    return weights


def moe(h, p, m):
    r = m["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    w = route(h @ p["router"].T, p["correction"], int(r["top"]), int(groups["count"]), int(groups["keep"]))
    y = torch.zeros_like(h)
    for e in range(int(r["experts"])):
        pe = {n: p[f"e{e}.{n}"] for n in ("gate", "up", "down")}
        y = y + w[:, e:e + 1] * gated_ff(h, pe)
    if m.get("shared") is not None:
        ps = {n: p[f"shared.{n}"] for n in ("gate", "up", "down")}
        y = y + torch.sigmoid(h @ p["shared.sg"].T) * gated_ff(h, ps)
    return y


def layer_runs(config):
    """(layer, does it open a pass of the loop other than the first), in the order the layers run."""
    n = len(config["layers"])
    loop = config.get("loop")
    if loop is None:
        return [(i, False) for i in range(n)]
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    runs = [(i, False) for i in range(start)]
    for k in range(times):
        runs += [(i, k > 0 and i == start) for i in range(start, stop)]
    return runs + [(i, False) for i in range(stop, n)]


def layer_tensors(tensors, prefix, dtype=F):
    return {k[len(prefix):]: v.to(dtype) for k, v in tensors.items() if k.startswith(prefix)}


def mixer(kind, h, p, m, eps):
    if kind == "attention":
        return rotary_attention(h, p, m, eps)
    if kind == "hgrn2":
        return hgrn2(h, p, m, eps)
    if kind == "parallel":
        left = window_attention(h, layer_tensors(p, "left.", h.dtype), m["left"], eps)
        right = mamba(h, layer_tensors(p, "right.", h.dtype), m["right"])
        return float(m["left_scale"]) * left + float(m["right_scale"]) * right
    raise ValueError(kind)


def forward(config, tensors, tokens, want_layers=False, dtype=F):
    """Logits [T, vocab] of one sequence (and the stream after every layer run, [runs, T, width])."""
    eps = float(config["norm"]["eps"])
    x0 = tensors["embed"].to(dtype)[torch.tensor(tokens)] * float(config["embedding"]["scale"])
    x, streams = x0, []
    for i, again in layer_runs(config):
        layer = config["layers"][i]
        p = layer_tensors(tensors, f"l{i}.", dtype)
        if again:
            x = x + x0
        h = input_conv(rms(x, eps) * p["norm1"], p["canon1"])
        x = x + mixer(layer["type"], h, layer_tensors(tensors, f"l{i}.mix.", dtype), layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + moe(rms(x, eps) * p["norm2"], layer_tensors(tensors, f"l{i}.mlp.", dtype), layer["mlp"])
        streams.append(x)
    logits = (rms(x, eps) * tensors["final.norm"].to(dtype)) @ tensors["head"].to(dtype).T
    if want_layers:
        return logits, torch.stack(streams)
    return logits


def greedy(config, tensors, prompt, n):
    """The n tokens that greedy decoding appends to the prompt."""
    tokens, out = list(prompt), []
    for _ in range(n):
        nxt = int(forward(config, tensors, tokens)[-1].argmax())
        tokens.append(nxt)
        out.append(nxt)
    return out
