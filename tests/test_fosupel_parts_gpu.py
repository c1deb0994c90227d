"""Every mechanism of Fosupel alone on the GPU against the plain functions, at sizes of its own: attention over a window and kept
first tokens whose heads mix their weights, retention, latent attention with a gate per column, xIELU, the router whose weights
stay as they are, the vector of a pass, the capped head and the block; and the kernels they added.  Requests run in portions
of many sizes beside one another; slots and pages are freed and used again (freed memory is NaN)."""
import pytest
import torch

from plain import fosupel_plain as P
from test_dimudra_parts_gpu import CUTS, DTYPES, EPS, LENGTHS, WIDTH, close, f64, i32, inputs, rebind, rows_of
from test_parts_gpu import cache_for, give_weights, runtime, step_in_portions

pytestmark = pytest.mark.gpu


def rope(dim, rot):
    from logssms_b200.config.specs import RopeSpec
    if rot is None:
        return None
    return RopeSpec(dim, rot[0], rot[1], 4096, (("factor", rot[2]),) if len(rot) > 2 else None, kind="rope_linear")


def plain_rot(rot):
    return None if rot is None else {"dims": rot[0], "base": rot[1], "scaling": {"factor": rot[2]} if len(rot) > 2 else None}


# --------------------------------------------------------------------------- attention with mixed weights
def talking_part(dtype, heads, kv_heads, dim, vdim, window, keep, rot, scale=0.3, seed=0, max_seq_len=256):
    from logssms_b200.config.specs import TalkingAttentionSpec
    from logssms_b200.parts import TalkingAttention
    part = TalkingAttention(TalkingAttentionSpec(WIDTH, heads, kv_heads, dim, vdim, scale, window=window, keep_first=keep, position=rope(dim, rot)))
    stored = give_weights(part, dtype, seed=seed)
    part.setup(runtime(dtype, max_seq_len=max_seq_len))
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": plain_rot(rot),
         "mask": None if window is None else {"size": window, "keep_first": keep}}
    return part, stored, m


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, window, keep, rot", [
    (6, 2, 16, 24, 20, 5, (8, 500.0, 3.0)), (4, 4, 32, 16, 33, 17, (32, 1e4)), (1, 1, 2, 1, 1, 1, None), (3, 3, 7, 9, 31, 3, (6, 9.0)),
    (4, 2, 10, 6, 64, 67, (4, 50.0, 2.5)), (18, 1, 16, 8, 16, 1, (16, 300.0)), (20, 4, 16, 8, 65, 64, (2, 7.0, 9.0)), (8, 2, 64, 128, 40, 20, (20, 1e6)),
    (16, 4, 128, 128, 30, 33, (64, 1e4, 4.0)), (6, 3, 48, 40, 2, 0, None), (12, 12, 16, 48, 17, 15, (16, 30.0)), (5, 1, 80, 72, None, 0, (10, 90.0)),
    (2, 1, 144, 160, 30, 4, (40, 1000.0)), (34, 17, 16, 16, 50, 12, None), (2, 2, 260, 24, 9, 2, None), (16, 16, 240, 64, 40, 16, (16, 30.0))])
def test_talking_attention_in_portions(dtype, heads, kv_heads, dim, vdim, window, keep, rot):
    scale = 1.2 * dim ** -0.5 * (3.0 if dtype == torch.float32 else 1.0)     # sharp: single keys carry the output
    part, stored, m = talking_part(dtype, heads, kv_heads, dim, vdim, window, keep, rot, scale, seed=heads + dim)
    cache, planner = cache_for([part.cache_needs()], dtype, max_requests=3)
    xs = inputs(LENGTHS, WIDTH, dtype, seed=1)
    for _ in range(2):                            # twice: the second time through slots and pages that were freed (and hold NaN)
        got = step_in_portions(planner, cache, LENGTHS, CUTS, lambda ctx, spans: part.forward(rows_of(xs, spans), ctx, 0))
        for x, y in zip(xs, got):
            close(y, P.window_attention(x.double(), f64(stored), m), dtype)


@pytest.mark.parametrize("dtype, dim", [(torch.float32, 4), (torch.float32, 16), (torch.bfloat16, 16)])
@pytest.mark.parametrize("window, keep", [(1, 0), (1, 1), (2, 3), (5, 16), (16, 15), (17, 17), (31, 33), (64, 1), (65, 64), (40, 20), (30, 90), (400, 5), (None, 0)])
@pytest.mark.parametrize("cuts", [[[200]], [[3], [2], [40], [2], [200]], [[50]] + [[1]] * 110, [[1]] * 40 + [[29], [200]]])
def test_outputs_name_the_keys_that_were_seen(dtype, dim, window, keep, cuts):
    """Queries of zero make all scores equal, a sink of -40 weighs nothing, the mix is the identity: the output is the mean of the
    seen values.  The values carry a one on every eighth token (per residue a column of its own), so every output counts the seen
    tokens of every residue: in prompts cut anywhere, in decoded tokens, over pages of 16, on the tensor cores (bfloat16) too."""
    n = 160
    part, stored, m = talking_part(dtype, 1, 1, dim, 8, window, keep, None, seed=3)
    for name in ("q", "v", "o"):
        stored[name] = torch.zeros_like(stored[name])
    for c in range(8):
        stored["v"][c, c] = 1.0                                  # value column c = input column c
        stored["o"][c, c] = 1.0
    stored["talk"], stored["sink"] = torch.ones_like(stored["talk"]), torch.full_like(stored["sink"], -40.0)
    rebind(part, stored, dtype)
    x = torch.zeros(n, WIDTH, dtype=dtype)
    x[torch.arange(n), torch.arange(n) % 8] = 1.0
    cache, planner = cache_for([part.cache_needs()], dtype, max_requests=2)
    (got,) = step_in_portions(planner, cache, [n], [[c[0]] for c in cuts], lambda ctx, spans: part.forward(rows_of([x], spans), ctx, 0))
    seen = P.seen_by(n, m["mask"]).double()
    total = seen.sum(1)
    counts = seen @ x[:, :8].double()                            # seen tokens of every residue
    have = got[:, :8].double() * total[:, None]
    # (a bfloat16 output of c / total is exact to 2^-9: the count of a residue is at most 20 here)
    assert float((have - counts).abs().max()) < (1e-3 if dtype == torch.float32 else 0.11), int((have - counts).abs().max(1).values.argmax())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window, keep", [(50, 6), (64, 5), (100, 0), (None, 0)])
def test_one_key_among_hundreds(dtype, window, keep):
    """600 tokens over pages of 16 whose late inputs are nearly a part of token 5's: with queries equal to keys the score of token 5 stands
    out.  A window that has passed it sees it as long as it is among the kept ones (and not a token longer), in a long prompt
    portion, a shorter one and decoded tokens."""
    n = 600
    part, stored, m = talking_part(dtype, 2, 1, 16, 8, window, keep, None, 0.6, seed=9, max_seq_len=640)
    stored["k"] = stored["q"][:16].clone()
    stored["q"] = torch.cat([stored["k"], stored["k"]], 0)
    rebind(part, stored, dtype)
    x = inputs([n], WIDTH, dtype, seed=4)[0]
    x[-40:] = 0.6 * x[5] + 0.05 * x[-40:]         # (each scores token 5 higher than itself)
    cache, planner = cache_for([part.cache_needs()], dtype, num_pages=48, max_requests=2, max_seq_len=640)
    cuts = [[400], [150], [10]] + [[1]] * 40
    (got,) = step_in_portions(planner, cache, [n], cuts, lambda ctx, spans: part.forward(rows_of([x], spans), ctx, 0))
    want = P.window_attention(x.double(), f64(stored), m)
    close(got, want, dtype)
    blind = x.clone()
    blind[5] = 0.0
    other = P.window_attention(blind.double(), f64(stored), m)
    moves = float((other[560] - want[560]).abs().max() / want[560].abs().max())
    assert moves > 0.05 if window is None or keep > 5 else moves == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, G, dim, vdim, window, keep", [(6, 2, 32, 24, 45, 20), (16, 4, 64, 128, 1 << 30, 0), (24, 6, 16, 104, 70, 70), (4, 4, 128, 160, 33, 1),
                                                           (3, 1, 12, 5, 20, 7), (16, 16, 32, 64, 100, 3)])
def test_talk_kernels_with_every_number_of_ranges(dtype, H, G, dim, vdim, window, keep):
    """The kernels alone: two requests over scattered pages, their tokens one by one with 1 to 9 key ranges (all of them, or a list
    of rows with holes), and in runs with 1 to 4."""
    from logssms_b200.ops import kernels as K
    g = torch.Generator().manual_seed(H + dim)
    lens, starts, page = [90, 33], [130, 0], 16
    pages = torch.randperm(24, generator=g).int()
    table = torch.full((2, 14), -1, dtype=torch.int32)
    table[0, :14] = pages[:14]
    table[1, :3] = pages[14:17]
    total = [s + n for s, n in zip(starts, lens)]
    ks = [torch.randn(t, G, dim, generator=g).to(dtype) for t in total]
    vs = [torch.randn(t, G, vdim, generator=g).to(dtype) for t in total]
    kc = torch.full((24, page, G, dim), float("nan"), dtype=dtype)
    vc = torch.full((24, page, G, vdim), float("nan"), dtype=dtype)
    for b in range(2):
        for j in range(total[b]):
            kc[int(table[b, j // page]), j % page], vc[int(table[b, j // page]), j % page] = ks[b][j], vs[b][j]
    if window < 130:                                                 # what no token of the step sees any more has gone
        for p in range(-(-keep // page), (130 - window + 1) // page):
            table[0, p] = -1
    T = sum(lens)
    q = torch.randn(T, H, dim, generator=g).to(dtype)
    talk, sinks = torch.randn(H, H, generator=g) * H ** -0.5, torch.randn(H, generator=g)
    scale = 1.5 * dim ** -0.5
    mask = None if window >= 1 << 30 else {"size": window, "keep_first": keep}
    want = []
    for b in range(2):
        qq = torch.zeros(total[b], H, dim, dtype=torch.float64)
        qq[starts[b]:] = q[sum(lens[:b]):sum(lens[:b + 1])].double()
        want.append(P.talking_attention(qq, ks[b].double(), vs[b].double(), scale, mask, sinks.double(), talk.double())[starts[b]:].reshape(lens[b], -1))
    want = torch.cat(want)
    req = torch.tensor([0] * lens[0] + [1] * lens[1], dtype=torch.int32).cuda()
    pos = torch.cat([torch.arange(s, s + n) for s, n in zip(starts, lens)]).int().cuda()
    args = (q.cuda(), kc.cuda(), vc.cuda(), table.cuda())
    tail = (talk.cuda(), scale, window, keep)
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    for splits in (1, 2, 3, 5, 9):
        close(K.talk_attention(*args, req, pos, *tail, 250, sinks=sinks.cuda(), splits=splits), want, dtype, tol)
    rows = [3, -1, 100, 90, 89, -1]
    out = torch.zeros(T, H * vdim, dtype=dtype).cuda()
    K.talk_attention(*args, req, pos, *tail, 250, token_list=i32(*rows), out=out, sinks=sinks.cuda())
    live = [r for r in rows if r >= 0]
    close(out[live], want[live], dtype, tol)
    assert float(out[[r for r in range(T) if r not in live]].abs().max()) == 0.0
    if dtype == torch.bfloat16 and K.talk_attention_tile_ok(args[0], args[2]):
        tiles = i32(*[v for b, n in enumerate(lens) for t0 in range(0, n, K.talk_tile_q()) for v in (b, t0)] + [-1, 0]).view(-1, 2)
        for splits in (1, 2, 4):
            out = torch.empty(T, H * vdim, dtype=dtype).cuda()
            K.talk_attention_tile(*args, i32(0, lens[0], T), i32(*starts), tiles, *tail, out, splits=splits, sinks=sinks.cuda())
            close(out, want, dtype, tol)
    no_sink = K.talk_attention(*args, req, pos, *tail, 250)
    assert float((no_sink.double().cpu() - want).abs().max()) > 1e-2 * float(want.abs().max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, G, dim, vdim, window, keep", [(4, 2, 32, 16, 20, 9), (3, 3, 16, 8, 40, 70), (2, 1, 12, 136, 17, 16)])
def test_window_attention_kernels_keep_first_tokens(dtype, H, G, dim, vdim, window, keep):
    """The kernels of the other designs' window attention with the option of kept first tokens, beside a bias by distance: a warp per
    row, key ranges, and runs on the tensor cores."""
    from logssms_b200.ops import kernels as K
    g = torch.Generator().manual_seed(dim)
    n, start, page = 70, 110, 16
    total = start + n
    table = torch.randperm(14, generator=g).int().view(1, 14)
    k, v = torch.randn(total, G, dim, generator=g).to(dtype), torch.randn(total, G, vdim, generator=g).to(dtype)
    kc, vc = torch.zeros(14, page, G, dim, dtype=dtype), torch.zeros(14, page, G, vdim, dtype=dtype)
    for j in range(total):
        kc[int(table[0, j // page]), j % page], vc[int(table[0, j // page]), j % page] = k[j], v[j]
    q = torch.randn(n, H, dim, generator=g).to(dtype)
    slopes, scale = torch.rand(H, generator=g) * 0.02, 1.5 * dim ** -0.5
    i = torch.arange(start, total)[:, None]
    j = torch.arange(total)[None]
    seen = P.seen_by(total, {"size": window, "keep_first": keep})[start:]
    s = torch.einsum("ihd,jhd->hij", q.double(), k.double().repeat_interleave(H // G, 1)) * scale - slopes.double()[:, None, None] * (i - j)
    w = torch.softmax(s.masked_fill(~seen, float("-inf")), -1)
    want = torch.einsum("hij,jhd->ihd", w, v.double().repeat_interleave(H // G, 1)).reshape(n, -1)
    pos = torch.arange(start, total).int().cuda()
    args = (q.cuda(), kc.cuda(), vc.cuda(), None, None, table.cuda(), None)
    opts = {"slopes": slopes.cuda(), "keep": keep}
    req = torch.zeros(n, dtype=torch.int32).cuda()
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    close(K.pooled_attention(*args, req, pos, None, scale, window, 0, **opts), want, dtype, tol)
    if K.pooled_attention_split_ok(args[0], args[2]):
        for splits in (1, 3):
            close(K.pooled_attention_split(*args, req, pos, None, scale, window, 0, splits, **opts), want, dtype, tol)
    if K.pooled_attention_tile_ok(args[0], args[2]):
        for splits in (1, 2):
            out = torch.empty(n, H * vdim, dtype=dtype).cuda()
            K.pooled_attention_tile(*args, i32(0, n), i32(start), pos, i32(0, 0, 0, 64).view(2, 2), None, scale, window, 0, out, splits=splits, **opts)
            close(out, want, dtype, tol)


# --------------------------------------------------------------------------- retention
def retention_part(dtype, heads, dim, vdim, rot, decay=None, seed=0, max_seq_len=256):
    from logssms_b200.config.specs import RetentionSpec
    from logssms_b200.parts import Retention
    decay = decay or [1.0 - 2.0 ** -(1 + 3 * h) for h in range(heads)]
    part = Retention(RetentionSpec(WIDTH, heads, dim, vdim, tuple(decay), EPS, position=rope(dim, rot)))
    stored = give_weights(part, dtype, seed=seed)
    part.setup(runtime(dtype, max_seq_len=max_seq_len))
    return part, stored, {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": plain_rot(rot)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dim, vdim, rot", [(3, 16, 24, (8, 40.0)), (2, 32, 40, (32, 1e4, 2.0)), (1, 1, 1, None), (4, 8, 16, (2, 5.0)), (2, 48, 72, None),
                                                   (3, 20, 5, (6, 50.0)), (1, 128, 32, (64, 1e6)), (2, 160, 8, (100, 1e4)), (1, 260, 12, (20, 9.0)), (2, 64, 64, (64, 1e4))])
def test_retention_in_portions(dtype, heads, dim, vdim, rot):
    part, stored, m = retention_part(dtype, heads, dim, vdim, rot, seed=heads + dim)
    cache, planner = cache_for([part.cache_needs()], dtype, max_requests=3)
    xs = inputs(LENGTHS, WIDTH, dtype, seed=1)
    for _ in range(2):
        got = step_in_portions(planner, cache, LENGTHS, CUTS, lambda ctx, spans: part.forward(rows_of(xs, spans), ctx, 0))
        for x, y in zip(xs, got):
            # (a head of one column is normed to its sign, where rounding decides)
            if vdim > 1 or dtype == torch.float32:
                close(y, P.retention(x.double(), f64(stored), m, EPS), dtype, 1e-3 if vdim == 1 else None)


@pytest.mark.parametrize("heads, dim, vdim, rot", [(1, 16, 24, (16, 1e4)), (2, 48, 8, (20, 60.0, 3.0)), (1, 256, 40, (256, 1e6))])
def test_retention_carries_the_state_through_segments(heads, dim, vdim, rot):
    """Long portions (segments of 256 tokens side by side in a bfloat16 engine) beside a short request, then decoded tokens; decays
    of 1 and of 0.3."""
    for dtype in DTYPES:
        part, stored, m = retention_part(dtype, heads, dim, vdim, rot, [1.0, 0.3][:heads], seed=dim, max_seq_len=1600)
        cache, planner = cache_for([part.cache_needs()], dtype, max_requests=3, max_seq_len=1600)
        lengths = [1100, 9, 530]
        xs = inputs(lengths, WIDTH, dtype, seed=2)
        got = step_in_portions(planner, cache, lengths, [[600, 2, 0], [413, 1, 520], [1, 1, 1], [84, 5, 2], [1, 0, 1], [1, 0, 6]],
                               lambda ctx, spans: part.forward(rows_of(xs, spans), ctx, 0))
        for x, y in zip(xs, got):
            close(y, P.retention(x.double(), f64(stored), m, EPS), dtype, 1e-4 if dtype == torch.float32 else None)


def test_retention_remembers_a_token_hundreds_of_steps_back():
    dtype = torch.float32
    part, stored, m = retention_part(dtype, 2, 16, 8, (8, 1e5), [1.0, 0.9995], seed=4, max_seq_len=1024)
    x = inputs([640], WIDTH, dtype, seed=3)[0] * 0.3
    x[5] *= 60.0
    cache, planner = cache_for([part.cache_needs()], dtype, max_requests=2, max_seq_len=1024)
    cuts = [[300], [1], [1], [2], [250]] + [[1]] * 86
    (got,) = step_in_portions(planner, cache, [640], cuts, lambda ctx, spans: part.forward(rows_of([x], spans), ctx, 0))
    want = P.retention(x.double(), f64(stored), m, EPS)
    close(got, want, dtype, 1e-4)
    blind = x.clone()
    blind[5] = 0.0
    other = P.retention(blind.double(), f64(stored), m, EPS)
    assert float((want - other)[-50:].abs().max() / want[-50:].abs().max()) > 0.05


@pytest.mark.parametrize("H, dk, dv, rot", [(2, 16, 24, 16), (1, 64, 40, 22), (2, 112, 9, 0), (1, 256, 32, 256)])
def test_rotated_chunks_are_sharper_than_bfloat16(H, dk, dv, rot):
    """Both kernels of the recurrence rotate q and k and scale k while they load them; the chunked one hands them and the state to the
    tensor cores as two bfloat16 terms each: outputs and states agree with the recurrence in float64 (from the same bfloat16
    rows) far closer than 8 bits of mantissa would."""
    from logssms_b200.ops import kernels as K
    from logssms_b200.parts.context import chunk_lists
    g = torch.Generator().manual_seed(dk)
    lens, starts = [70, 41], [0, 50]
    T = sum(lens)
    qkv = torch.randn(T, H * (2 * dk + dv) + 3, generator=g).bfloat16()
    handed = torch.randn(H, dk, dv, generator=g)
    decay = torch.tensor([0.97, 1.0][:H])
    pos = torch.cat([torch.arange(s, s + n) for s, n in zip(starts, lens)])
    r = {"dims": rot, "base": 300.0} if rot else None
    f = torch.tensor([300.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float64)
    angle = torch.arange(128, dtype=torch.float64)[:, None] * f
    table = torch.cat([torch.cos(angle), torch.sin(angle)], 1).float().cuda().contiguous()
    k_scale = dk ** -0.5
    x = qkv.double()
    q = P.rotate_halves(x[:, :H * dk].view(T, H, dk), pos, r)
    k = P.rotate_halves(x[:, H * dk:2 * H * dk].view(T, H, dk), pos, r) * k_scale
    v = x[:, 2 * H * dk:H * (2 * dk + dv)].view(T, H, dv)
    want, states = [], []
    for lo, hi, S0 in ((0, 70, torch.zeros(H, dk, dv)), (70, T, handed)):
        S = S0.double()
        for t in range(lo, hi):
            S = decay.double()[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
            want.append((q[t][:, :, None] * S).sum(1).reshape(-1))
        states.append(S)
    want = torch.stack(want)
    chunks, per_request = chunk_lists(lens, K.GLA_CHUNK)
    opts = {"head_decay": decay.cuda(), "turn": table, "positions": pos.int().cuda(), "k_scale": k_scale}
    for kernel in ("chunked", "scan"):
        state = torch.full((3, H, dk, dv), float("nan"))
        state[2] = handed
        state = state.cuda()
        where = (i32(0, 70, T), i32(*starts), i32(0, 2))
        if kernel == "chunked":
            o = torch.empty(T, H * dv, device="cuda")
            K.gla_chunked(qkv.cuda(), None, state, *where, torch.from_numpy(chunks).cuda(), chunks.shape[0], torch.from_numpy(per_request).cuda(),
                          per_request.shape[0], H, dk, dv, 1.0, 1.0, out=o, two_terms=True, **opts)
        else:
            o = K.gla_scan(qkv.cuda(), None, state, *where, 2, H, dk, dv, 1.0, 1.0, **opts)
        close(o, want, torch.float32, 5e-5)
        close(state[0], states[0], torch.float32, 5e-5)
        close(state[2], states[1], torch.float32, 5e-5)


# --------------------------------------------------------------------------- latent attention
def latent_part(dtype, heads, dim, rot_dim, vdim, rank, rot, scale=0.25, seed=0, max_seq_len=256):
    from logssms_b200.config.specs import LatentAttentionSpec
    from logssms_b200.parts import LatentAttention
    part = LatentAttention(LatentAttentionSpec(WIDTH, heads, dim, rot_dim, vdim, rank, scale, None, rope(rot_dim, rot), EPS, pairing="neighbours",
                                               sink=True, column_gate=True), perturb_init=True)
    stored = give_weights(part, dtype, seed=seed)
    part.setup(runtime(dtype, max_seq_len=max_seq_len))
    return part, stored, {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": plain_rot(rot)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dim, rot_dim, vdim, rank, rot", [
    (4, 16, 8, 24, 40, (8, 1000.0)), (8, 32, 16, 32, 64, (16, 1e5)), (1, 2, 0, 1, 1, None), (3, 10, 6, 7, 20, (6, 50.0)), (16, 24, 32, 16, 128, (32, 1e4)),
    (2, 64, 16, 64, 256, (16, 10.0, 2.0)), (5, 8, 16, 6, 32, (16, 300.0)), (20, 16, 16, 16, 96, (16, 1e6))])
def test_latent_attention_with_a_gate_per_column(dtype, heads, dim, rot_dim, vdim, rank, rot):
    scale = 0.25 * (3.0 if dtype == torch.float32 else 1.0)
    part, stored, m = latent_part(dtype, heads, dim, rot_dim, vdim, rank, rot, scale, seed=heads + rank)
    cache, planner = cache_for([part.cache_needs()], dtype, max_requests=3)
    xs = inputs(LENGTHS, WIDTH, dtype, seed=1)
    for _ in range(2):
        got = step_in_portions(planner, cache, LENGTHS, CUTS, lambda ctx, spans: part.forward(rows_of(xs, spans), ctx, 0))
        for x, y in zip(xs, got):
            close(y, P.latent_attention(x.double(), f64(stored), m, EPS), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T, H, K_, N", [(3, 4, 32, 24), (33, 2, 16, 6), (90, 3, 40, 7), (200, 8, 64, 64), (40, 1, 8, 1)])
def test_heads_product_with_a_gate(dtype, T, H, K_, N):
    """The per-head product with a gate per output column: in the kernel's epilogue, and behind the library's product (many rows)."""
    from logssms_b200.ops import kernels as K
    g = torch.Generator().manual_seed(T)
    a, w = torch.randn(T, H, K_ + 3, generator=g).to(dtype)[:, :, :K_], (torch.randn(H, K_, N, generator=g) * K_ ** -0.5).to(dtype)
    gate = torch.randn(T, 5 + H * N + 1, generator=g).to(dtype)
    for shift in (4, 5):                                          # column views that are and are not aligned to pairs
        view = gate[:, shift:shift + H * N]
        want = torch.einsum("thk,hkn->thn", a.double(), w.double()) * torch.sigmoid(view.double()).view(T, H, N)
        got = K.heads_matmul(a.cuda(), w.cuda(), gate=gate.cuda()[:, shift:shift + H * N])
        close(got, want, dtype, 1e-5 if dtype == torch.float32 else 1.5e-2)


# --------------------------------------------------------------------------- feed-forwards
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff", [1, 24, 72, 37])
def test_dense_layer_with_xielu(dtype, ff):
    from logssms_b200.config.specs import DenseMLPSpec
    from logssms_b200.parts import DenseMLP
    part = DenseMLP(DenseMLPSpec(WIDTH, ff, "xielu"))
    stored = give_weights(part, dtype, seed=ff)
    for p, q in ((0.0, 0.0), (2.5, -3.0), (-2.0, 1.7)):
        stored["act"] = torch.tensor([p, q]).to(dtype)
        rebind(part, stored, dtype)
        for n in (1, 5, 90):
            (x,) = inputs([n], WIDTH, dtype, seed=n)
            close(part.forward(x.cuda()), P.dense_ff(x.double(), f64(stored)), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_xielu_kernel_at_large_and_tiny_values(dtype):
    from logssms_b200.ops import kernels as K
    z = torch.tensor([0.0, -0.0, 1e-6, -1e-6, 1e-3, -1e-3, 0.3, -0.3, 5.0, -5.0, 40.0, -90.0, -200.0, 7.0, -0.05, 2.0]).to(dtype)
    a, b = 0.8, 1.3
    for n in (16, 13):
        want = P.xielu(z[:n].double(), torch.tensor(0.8, dtype=torch.float64).expm1().log(), torch.tensor(0.8, dtype=torch.float64).expm1().log())
        got = K.xielu(z[:n].cuda(), torch.tensor([a, b]).cuda())
        assert torch.allclose(got.double().cpu(), want, rtol=2e-6 if dtype == torch.float32 else 5e-3, atol=1e-12)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts, top, ff, shared", [(12, 3, 16, 24), (6, 2, 22, 14), (1, 1, 8, 1), (10, 10, 7, 9), (40, 5, 8, None), (4, 2, 32, None)])
def test_routed_feed_forward(dtype, experts, top, ff, shared):
    """The chosen experts weigh what the softmax over all experts gives them; the shared expert has a gate per token, or is absent."""
    from logssms_b200.config import make_model_config
    from logssms_b200.parts import RoutedMLP
    from tiny_fosupel import latent, model, moe
    m = moe(experts, top if dtype == torch.float32 else experts, ff, shared)
    raw = model(WIDTH, 50, EPS, 1.0, 9.0, None, [{**latent(1, 2, 0, 1, 1, 0.5), "mlp": m}])
    part = RoutedMLP(make_model_config(raw).model_spec().layers[0].feed_forward)
    stored = give_weights(part, dtype, seed=experts)
    for n in (1, 5, 90, 600):                                     # from 592 tokens on a CTA of the router takes four of them
        (x,) = inputs([n], WIDTH, dtype, seed=n)
        close(part.forward(x.cuda()), P.moe(x.double(), f64(stored), m), dtype)


# --------------------------------------------------------------------------- stream, head, block
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [24, 31, 1030])
def test_stream_sum_with_a_vector_for_every_row(dtype, width):
    from logssms_b200.ops import kernels as K
    g = torch.Generator().manual_seed(width)
    x, row, w = torch.randn(5, width, generator=g), torch.randn(width, generator=g), torch.randn(width, generator=g)
    ys = [torch.randn(5, width, generator=g).to(dtype) for _ in range(2)]
    for addends in ([], list(zip(ys, (0.7, -1.3)))):
        new = x.double() + sum(s * y.double() for y, s in addends) + row.double()
        xs = x.cuda()
        _, h = K.stream_add_many(xs, [(y.cuda(), s) for y, s in addends], w.cuda(), EPS, "rmsnorm", dtype, row=row.cuda())
        close(xs, new, torch.float32, 1e-6)
        close(h, P.rms(new, EPS) * w.double(), dtype, 1e-5 if dtype == torch.float32 else 1e-2)
        xs = x.cuda()
        cw = torch.randn(width, 1, generator=g)
        h = K.stream_add_conv_step(xs, [(y.cuda(), s) for y, s in addends], w.cuda(), EPS, "rmsnorm", cw.cuda(), None, i32(*range(5)), i32(*range(5)), dtype,
                                   row=row.cuda())
        close(xs, new, torch.float32, 1e-6)
        close(h, P.rms(new, EPS) * w.double() * cw[:, 0].double(), dtype, 1e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_capped_head_is_the_embedding(dtype):
    from logssms_b200.parts import SoftcapLMHead, StreamEmbedding
    embedding = StreamEmbedding(77, WIDTH)
    stored = give_weights(embedding, dtype, seed=1)
    head = SoftcapLMHead(77, WIDTH, 1.0, embedding, cap=4.0)
    assert head.param_specs() == {}
    for n in (1, 3, 50):
        (h,) = inputs([n], WIDTH, dtype, seed=n)
        got = head.forward(h.cuda())
        assert got.dtype == torch.float32
        close(got, 4.0 * torch.tanh(h.double() @ stored["embed"].double().T / 4.0), torch.float32, 1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind, ff, mult", [("pair", "dense", 0.6), ("latent", "moe", 1.0), ("pair", None, -1.2), ("latent", "dense", 0.3), ("pair", "moe", 1.0)])
def test_block_in_portions(dtype, kind, ff, mult):
    """The block with its residual factor, a mixer of one or two branches, with and without a feed-forward, on a 32-bit stream."""
    from logssms_b200.config import make_model_config
    from logssms_b200.ops import kernels as K
    from logssms_b200.parts import PreNormStreamBlock
    from tiny_fosupel import dense, latent, left, model, moe, parallel, right
    layer = latent(4, 16, 16, 8, 32, 0.3) if kind == "latent" else parallel(left(4, 2, 16, 8, 21, 6, 0.4, (8, 99.0, 2.0)), right(2, 16, 24, (16, 50.0)), 1.2, 0.7)
    mlp = {"dense": dense(40), "moe": moe(6, 6, 16, 8), None: None}[ff]
    raw = model(WIDTH, 50, EPS, mult, 9.0, None, [{**layer, "mlp": mlp}])
    block = PreNormStreamBlock(make_model_config(raw).model_spec().layers[0], perturb_init=True)
    stored = give_weights(block, dtype, seed=5)
    block.setup(runtime(dtype))
    cache, planner = cache_for([block.cache_needs()], dtype, max_requests=3)
    xs = inputs(LENGTHS, WIDTH, dtype, seed=8)

    def run(ctx, spans):
        rows = rows_of(xs, spans)
        out, rest = block.forward(K.StreamRows(rows.float().clone(), rows), None, ctx, 0)
        assert rest is None and out.f32.dtype == torch.float32
        return out.f32
    for _ in range(2):
        got = step_in_portions(planner, cache, LENGTHS, CUTS, run)
        w = f64(stored)
        part = lambda prefix: {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}
        for x, y in zip(xs, got):
            want = x.double()
            want = want + mult * P.mixer(layer["type"], P.rms(want, EPS) * w["norm1"], part("mix."), layer["mixer"], EPS)
            if ff:
                h = P.rms(want, EPS) * w["norm2"]
                want = want + mult * (P.dense_ff(h, part("mlp.")) if ff == "dense" else P.moe(h, part("mlp."), mlp))
            close(y, want, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_stream_after_every_layer_run(tmp_path, name, dtype):
    """The stream after every run of every layer (a looped layer once per pass, before the next pass's vector is added), which the
    engine shows to `layer_tap`, and the same logits with and without the tap (the vector then joins in a closing kernel)."""
    from logssms_b200.engine import Engine, StepEntry
    from tiny_fosupel import FOSU, make_fosupel_dir, read_folder
    raw = FOSU[name]
    folder = make_fosupel_dir(tmp_path / "m", raw, seed=3, dtype=torch.float32 if dtype == "float32" else torch.bfloat16, calm=dtype == "bfloat16")
    ids = [int(i) for i in torch.randint(0, raw["vocab"], (37,), generator=torch.Generator().manual_seed(2))]
    config, tensors = read_folder(folder)
    logits, streams = P.forward(config, tensors, ids, want_layers=True)
    engine = Engine(folder, dtype, max_requests=2, max_seq_len=64, num_pages=2, use_graphs=False)
    seen = []
    engine.layer_tap = lambda i, x, residual: seen.append(x.f32.clone())
    r = engine.new_request()
    a = engine.step([StepEntry(r, ids, list(range(len(ids))))]).clone()
    engine.release(r)
    assert len(seen) == streams.shape[0] == len(P.layer_runs(raw))
    tol = 2e-5 if dtype == "float32" else 6e-2
    for i, s in enumerate(seen):
        err = (s.double().cpu() - streams[i]).pow(2).mean().sqrt() / streams[i].pow(2).mean().sqrt()
        assert float(err) < tol, (i, float(err))
    engine.layer_tap = None
    r = engine.new_request()
    b = engine.step([StepEntry(r, ids, list(range(len(ids))))])
    close(b, a, torch.float32, 1e-5 if dtype == "float32" else 2e-2)
    if dtype == "float32":
        close(a, logits, torch.float32, 1e-4)
