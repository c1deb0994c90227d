"""A plain, slow Fosupel: one function per mechanism, written from the design's equations in float64 tensor operations,
token by token where the design is a recurrence.  It shares no code with the engine; the engine's tests compare against it.

A model is (config mapping, {tensor name: tensor}); a request is a list of token ids.  `forward` returns the logits at
every position and, on request, the stream after every layer run.  With another `dtype` than float64 every tensor and every
intermediate result is of that dtype (angles excepted): what rounding alone does to a model.
"""
from __future__ import annotations

import torch

F = torch.float64
silu = torch.nn.functional.silu
softplus = torch.nn.functional.softplus


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def angles(positions, rot, dtype):
    """cos and sin [T, 1, dims/2] of position * base^(-2i/dims) / factor (the factor of a linear scaling, or 1)."""
    dims, base = int(rot["dims"]), float(rot["base"])
    factor = float(rot["scaling"]["factor"]) if rot.get("scaling") else 1.0
    f = torch.tensor([base ** (-2.0 * i / dims) / factor for i in range(dims // 2)], dtype=F)
    a = positions.to(F)[:, None] * f[None, :]
    return torch.cos(a)[:, None, :].to(dtype), torch.sin(a)[:, None, :].to(dtype)


def rotate_halves(x, positions, rot):
    """x [T, heads, d]: of every head's first rot.dims columns, column i pairs with column i + dims/2 (`rot` None: none turn)."""
    if rot is None:
        return x
    dims = int(rot["dims"])
    half = dims // 2
    cos, sin = angles(positions, rot, x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], -1)


def rotate_neighbours(x, positions, rot):
    """The same with column 2i paired with column 2i + 1."""
    if rot is None:
        return x
    dims = int(rot["dims"])
    cos, sin = angles(positions, rot, x.dtype)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def seen_by(T, mask):
    """[T, T] booleans: does position i see j?  mask: {size, keep_first} or None (every j <= i)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    if mask is None:
        return j <= i
    return (j <= i) & ((i - j < int(mask["size"])) | (j < int(mask.get("keep_first", 0))))


def sink_softmax(s, seen, sink):
    """s [H, T, T] scores, sink [H]: e^s / (sum of e^s over what is seen + e^sink)."""
    s = s.masked_fill(~seen[None], float("-inf"))
    m = torch.maximum(s.amax(-1, keepdim=True), sink[:, None, None])
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - m))


def talking_attention(q, k, v, scale, mask, sink, talk):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: query head h scores the keys of key/value head h // (H / G); the heads' softmax
    weights are mixed by talk [H, H], then every head applies its mixed weights to the values of its own key/value head."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    w = sink_softmax(torch.einsum("ihd,jhd->hij", q, k) * scale, seen_by(T, mask), sink)
    return torch.einsum("hij,jhd->ihd", torch.einsum("hg,gij->hij", talk, w), v)


def window_attention(h, p, m):
    """The left branch of a 'parallel' mixer."""
    T, H, G, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(T)
    q = rotate_halves((h @ p["q"].T).view(T, H, d), pos, m.get("rot"))
    k = rotate_halves((h @ p["k"].T).view(T, G, d), pos, m.get("rot"))
    v = (h @ p["v"].T).view(T, G, dv)
    return talking_attention(q, k, v, float(m["scale"]), m.get("mask"), p["sink"], p["talk"]).reshape(T, H * dv) @ p["o"].T


def decayed_memory(q, k, v, decay):
    """q, k [T, H, d], v [T, H, dv], decay [H]: S <- decay_h S + k v^T, o = S^T q, from S = 0."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    o = torch.zeros_like(v)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (q[t][:, :, None] * S).sum(1)
    return o


def retention(h, p, m, eps):
    """The right branch of a 'parallel' mixer."""
    T, H, d, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(T)
    q = rotate_halves((h @ p["q"].T).view(T, H, d), pos, m.get("rot"))
    k = rotate_halves((h @ p["k"].T).view(T, H, d), pos, m.get("rot")) * d ** -0.5
    v = (h @ p["v"].T).view(T, H, dv)
    o = rms(decayed_memory(q, k, v, torch.tensor(m["decay"], dtype=h.dtype)), eps).reshape(T, H * dv)
    return (o * silu(h @ p["g"].T)) @ p["o"].T


def latent_attention(h, p, m, eps):
    T, H, d, r = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["rot_dim"])
    dv, rank = int(m["vdim"]), int(m["kv_rank"])
    pos = torch.arange(T)
    q = (h @ p["q"].T).view(T, H, d + r)
    down = h @ p["dkv"].T
    c = rms(down[:, :rank], eps) * p["dkv.norm"]
    key_part = rotate_neighbours(down[:, None, rank:], pos, m.get("rot"))
    k = torch.cat([(c @ p["uk"].T).view(T, H, d), key_part.expand(T, H, r)], -1)
    q = torch.cat([q[..., :d], rotate_neighbours(q[..., d:], pos, m.get("rot"))], -1)
    v = (c @ p["uv"].T).view(T, H, dv)
    w = sink_softmax(torch.einsum("ihd,jhd->hij", q, k) * float(m["scale"]), seen_by(T, None), p["sink"])
    o = torch.einsum("hij,jhd->ihd", w, v).reshape(T, H * dv)
    return (o * torch.sigmoid(h @ p["g"].T)) @ p["o"].T


def xielu(z, p, q):
    """softplus(p) z^2 + z/2 above zero, (1/2 + softplus(q)) (e^z - 1 - z) + z/2 below."""
    return torch.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (torch.expm1(z.clamp_max(0)) - z)) + 0.5 * z


def dense_ff(h, p):
    return xielu(h @ p["up"].T, p["act"][0], p["act"][1]) @ p["down"].T


def gated_ff(h, p):
    return (silu(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def route(z, top):
    """Router outputs z [T, n] -> weights [T, n] (0: not chosen): the `top` largest of the softmax over all outputs, as they are."""
    s = torch.softmax(z, -1)
    keep = torch.zeros_like(s).scatter_(1, s.topk(top, -1).indices, 1.0)
    return s * keep


def moe(h, p, m):
    r = m["router"]
    w = route(h @ p["router"].T, int(r["top"]))
    y = torch.zeros_like(h)
    for e in range(int(r["experts"])):
        y = y + w[:, e:e + 1] * gated_ff(h, {n: p[f"e{e}.{n}"] for n in ("gate", "up", "down")})
    if m.get("shared") is not None:
        y = y + torch.sigmoid(h @ p["shared.sg"].T) * gated_ff(h, {n: p[f"shared.{n}"] for n in ("gate", "up", "down")})
    return y


def layer_runs(config):
    """(layer, number of the loop's pass that opens right before it or None), in the order the layers run."""
    n = len(config["layers"])
    loop = config.get("loop")
    if loop is None:
        return [(i, None) for i in range(n)]
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    runs = [(i, None) for i in range(start)]
    for k in range(times):
        runs += [(i, k if i == start else None) for i in range(start, stop)]
    return runs + [(i, None) for i in range(stop, n)]


def layer_tensors(tensors, prefix, dtype=F):
    return {k[len(prefix):]: v.to(dtype) for k, v in tensors.items() if k.startswith(prefix)}


def mixer(kind, h, p, m, eps):
    if kind == "latent_attention":
        return latent_attention(h, p, m, eps)
    if kind == "parallel":
        left = window_attention(h, layer_tensors(p, "left.", h.dtype), m["left"])
        right = retention(h, layer_tensors(p, "right.", h.dtype), m["right"], eps)
        return float(m["left_scale"]) * left + float(m["right_scale"]) * right
    raise ValueError(kind)


def forward(config, tensors, tokens, want_layers=False, dtype=F):
    """Logits [T, vocab] of one sequence (and the stream after every layer run, [runs, T, width])."""
    eps, mult = float(config["norm"]["eps"]), float(config["residual_mult"])
    embed = tensors["embed"].to(dtype)
    x, streams = embed[torch.tensor(tokens)], []
    for i, turn in layer_runs(config):
        layer = config["layers"][i]
        p = layer_tensors(tensors, f"l{i}.", dtype)
        if turn is not None:
            x = x + tensors["loop.step"][turn].to(dtype)
        h = rms(x, eps) * p["norm1"]
        x = x + mult * mixer(layer["type"], h, layer_tensors(tensors, f"l{i}.mix.", dtype), layer["mixer"], eps)
        if layer.get("mlp") is not None:
            h = rms(x, eps) * p["norm2"]
            ff = layer_tensors(tensors, f"l{i}.mlp.", dtype)
            x = x + mult * (dense_ff(h, ff) if layer["mlp"]["kind"] == "dense" else moe(h, ff, layer["mlp"]))
        streams.append(x)
    cap = float(config["logit_softcap"])
    logits = cap * torch.tanh((rms(x, eps) * tensors["final.norm"].to(dtype)) @ embed.T / cap)
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
