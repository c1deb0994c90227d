"""Every mechanism of Dimudra alone on the GPU against the plain functions, at sizes of its own: gated attention (over a window
with whole-row norms and biases; rotary with unit heads and one added to the denominator), the selective scan, linear attention
whose forget gate decides what is written, the router with groups ranked by their best pair and the gated shared expert, the input
convolution, and the block; and the kernels they added.  Requests run in portions of many sizes beside one another; slots and
pages are freed and used again (freed memory is NaN)."""
import math

import pytest
import torch

from plain import dimudra_plain as P
from tiny_dimudra import calm_routers
from test_parts_gpu import cache_for, give_weights, runtime, step_in_portions

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
TOL = {torch.float32: 3e-5, torch.bfloat16: 3e-2}
CUTS = [[37, 0, 9], [5, 20, 1], [1, 1, 1], [2, 3, 1], [64, 2, 1], [1, 30, 2], [200, 200, 200]]
LENGTHS = [130, 61, 40]
WIDTH = 56
EPS = 1e-5


def close(got, want, dtype, tol=None):
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape, (got.shape, want.shape)
    assert torch.isfinite(got).all()
    err = float((got - want).abs().max() / want.abs().max().clamp_min(1e-30))
    assert err <= (tol or TOL[dtype]), f"error {err:.3g}"


def inputs(lengths, width, dtype, seed=0):
    g = torch.Generator().manual_seed(seed)
    return [torch.randn(n, width, generator=g).to(dtype) for n in lengths]


def rows_of(xs, spans):
    return torch.cat([xs[r][lo:hi] for r, lo, hi in spans]).cuda()


def f64(stored):
    return {k: v.double() for k, v in stored.items()}


def rebind(part, stored, dtype):
    from logssms_b200.weights.loader import check_and_place
    part.bind_tree(check_and_place(part, {k: v.to(dtype) for k, v in stored.items()}, dtype, "cuda"))


def i32(*v):
    return torch.tensor(v, dtype=torch.int32).cuda()


# --------------------------------------------------------------------------- gated attention
def attention_part(dtype, heads, kv_heads, dim, vdim, *, window=None, rot=None, row=False, scale=0.3, seed=0, max_seq_len=256):
    """row True: the windowed branch (biases, whole-row norms); False: the rotary mixer (unit heads, one added)."""
    from logssms_b200.config.specs import GatedAttentionSpec, RopeSpec
    from logssms_b200.parts import GatedAttention
    position = None if rot is None else RopeSpec(dim, rot[0], rot[1], 4096, kind="rope_ramp")
    spec = GatedAttentionSpec(WIDTH, heads, kv_heads, dim, vdim, scale, EPS, window=window, position=position, proj_bias=row,
                              qk_norm="row" if row else "head_unit", sink_zero=not row)
    part = GatedAttention(spec, perturb_init=True)
    stored = give_weights(part, dtype, seed=seed)
    part.setup(runtime(dtype, max_seq_len=max_seq_len))
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return part, stored, m


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, window", [
    (6, 2, 16, 24, 20), (4, 1, 32, 32, 70), (2, 2, 16, 8, 1), (1, 1, 2, 1, 2), (4, 2, 10, 6, 64), (3, 3, 40, 16, 17), (8, 2, 64, 128, 33),
    (5, 1, 7, 9, 16), (2, 1, 144, 160, 30), (2, 1, 24, 16, None)])
def test_windowed_attention_in_portions(dtype, heads, kv_heads, dim, vdim, window):
    scale = 1.2 * dim ** -0.5 * (3.0 if dtype == torch.float32 else 1.0)     # sharp: single keys carry the output
    part, stored, m = attention_part(dtype, heads, kv_heads, dim, vdim, window=window, row=True, scale=scale, seed=heads + dim)
    cache, planner = cache_for([part.cache_needs()], dtype, max_requests=3)
    xs = inputs(LENGTHS, WIDTH, dtype, seed=1)
    for _ in range(2):                            # twice: the second time through slots and pages that were freed (and hold NaN)
        got = step_in_portions(planner, cache, LENGTHS, CUTS, lambda ctx, spans: part.forward(rows_of(xs, spans), ctx, 0))
        for x, y in zip(xs, got):
            close(y, P.window_attention(x.double(), f64(stored), m, EPS), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, rot", [
    (4, 2, 16, 8, (8, 500.0)), (4, 4, 32, 32, (32, 10000.0)), (1, 1, 2, 1, (2, 100.0)), (3, 1, 22, 18, None), (6, 2, 24, 40, (6, 30.0)),
    (8, 2, 64, 64, (20, 30000.0)), (2, 1, 9, 5, (4, 9.0)), (2, 2, 128, 96, (64, 1e6)), (1, 1, 160, 200, (40, 1000.0))])
def test_rotary_attention_in_portions(dtype, heads, kv_heads, dim, vdim, rot):
    scale = 1.2 * dim ** -0.5 * (3.0 if dtype == torch.float32 else 1.0)
    part, stored, m = attention_part(dtype, heads, kv_heads, dim, vdim, rot=rot, scale=scale, seed=heads + dim)
    cache, planner = cache_for([part.cache_needs()], dtype, max_requests=3)
    xs = inputs(LENGTHS, WIDTH, dtype, seed=2)
    for _ in range(2):
        got = step_in_portions(planner, cache, LENGTHS, CUTS, lambda ctx, spans: part.forward(rows_of(xs, spans), ctx, 0))
        for x, y in zip(xs, got):
            close(y, P.rotary_attention(x.double(), f64(stored), m, EPS), dtype)


@pytest.mark.parametrize("row, window", [(True, 1), (True, 2), (True, 5), (True, 16), (True, 17), (True, 31), (True, 64), (True, 65), (False, None)])
@pytest.mark.parametrize("cuts", [[[200]], [[3], [2], [40], [2], [200]], [[50]] + [[1]] * 110, [[1]] * 40 + [[29], [200]]])
def test_outputs_name_the_keys_that_were_seen(row, window, cuts):
    """Queries of zero make all scores equal: the output is the sum of the seen values over their number (plus one where one is
    added to the denominator).  The values carry a one and the token's position, so every output names how many keys were seen and
    which: in prompts cut anywhere, in decoded tokens, over pages of 16."""
    dtype = torch.float32
    n, dim = 160, 4
    part, stored, m = attention_part(dtype, 1, 1, dim, dim, window=window, row=row, seed=3)
    stored["q"] = torch.zeros_like(stored["q"])
    stored["v"] = torch.zeros_like(stored["v"])
    stored["v"][0, 0] = 1.0                                  # value column 0 = input column 0 (a one), column 1 = column 1 (the position)
    stored["v"][1, 1] = 1.0
    stored["g"] = torch.zeros_like(stored["g"])              # gate: sigmoid(0) = 1/2
    stored["o"] = torch.zeros_like(stored["o"])
    stored["o"][0, 0] = 1.0
    stored["o"][1, 1] = 1.0
    if row:
        stored["q.b"], stored["v.b"] = torch.zeros_like(stored["q.b"]), torch.zeros_like(stored["v.b"])
    rebind(part, stored, dtype)
    x = torch.zeros(n, WIDTH)
    x[:, 0] = 1.0
    x[:, 1] = torch.arange(n, dtype=torch.float32)
    cache, planner = cache_for([part.cache_needs()], dtype, max_requests=2)
    (got,) = step_in_portions(planner, cache, [n], [[c[0]] for c in cuts], lambda ctx, spans: part.forward(rows_of([x], spans), ctx, 0))
    for i in range(n):
        count = i + 1 if window is None else min(window, i + 1)
        first = i - count + 1
        below = count + (0 if row else 1)
        want_one, want_pos = 0.5 * count / below, 0.5 * sum(range(first, i + 1)) / below
        assert abs(float(got[i, 0]) - want_one) < 1e-5 and abs(float(got[i, 1]) - want_pos) < 1e-3 * max(1.0, want_pos), \
            f"position {i}: saw {float(got[i, 0]):.6f}, {float(got[i, 1]):.4f}; {count} keys from {first} give {want_one:.6f}, {want_pos:.4f}"


@pytest.mark.parametrize("window", [33, 64, 65])
def test_outputs_name_the_keys_on_the_tensor_cores_too(window):
    """The same in bfloat16, whose prompt portions run on the tensor cores: the seen tokens' number from values of one."""
    dtype = torch.bfloat16
    n, dim = 160, 16
    part, stored, m = attention_part(dtype, 1, 1, dim, dim, window=window, row=True, seed=3)
    for name in ("q", "v", "g", "o", "q.b", "v.b"):
        stored[name] = torch.zeros_like(stored[name])
    stored["v"][0, 0] = 1.0
    stored["v"][1, 1] = 1.0                                  # column 1: a one on one token in a hundred, zero elsewhere
    stored["o"][0, 0] = 1.0
    stored["o"][1, 1] = 1.0
    rebind(part, stored, dtype)
    for marked in (0, 15, 16, 63, 64, 100):
        x = torch.zeros(n, WIDTH, dtype=dtype)
        x[:, 0] = 1.0
        x[marked, 1] = 1.0
        cache, planner = cache_for([part.cache_needs()], dtype, max_requests=2)
        (got,) = step_in_portions(planner, cache, [n], [[70], [2], [60], [1], [40]], lambda ctx, spans: part.forward(rows_of([x], spans), ctx, 0))
        for i in range(n):
            seen = marked <= i < marked + window
            want = 0.5 / min(window, i + 1) if seen else 0.0
            assert abs(float(got[i, 0]) - 0.5) < 4e-3 and abs(float(got[i, 1]) - want) <= 5e-3 * max(want, 1e-3) + (0 if seen else 1e-9), (marked, i)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_key_far_back_among_hundreds(dtype):
    """600 tokens over pages of 16 whose last 40 inputs are nearly token 5's: with queries equal to keys the score of token 5
    stands out, in a long prompt portion, a shorter one and decoded tokens."""
    n = 600
    part, stored, m = attention_part(dtype, 2, 1, 16, 8, scale=0.6, seed=9, max_seq_len=640)
    stored["k"] = stored["q"][:16].clone()
    stored["q"] = torch.cat([stored["k"], stored["k"]], 0)
    rebind(part, stored, dtype)
    x = inputs([n], WIDTH, dtype, seed=4)[0]
    x[-40:] = x[5] + 0.05 * x[-40:]
    cache, planner = cache_for([part.cache_needs()], dtype, num_pages=48, max_requests=2, max_seq_len=640)
    cuts = [[400], [150], [10]] + [[1]] * 40
    (got,) = step_in_portions(planner, cache, [n], cuts, lambda ctx, spans: part.forward(rows_of([x], spans), ctx, 0))
    want = P.rotary_attention(x.double(), f64(stored), m, EPS)
    close(got, want, dtype)
    blind = x.clone()
    blind[5] = 0.0
    other = P.rotary_attention(blind.double(), f64(stored), m, EPS)
    assert float((other[560] - want[560]).abs().max()) > 0.05 * float(want[560].abs().max())    # token 5 matters to the first late query


@pytest.mark.parametrize("norm", ["none", "row", "head"])
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, rot", [(3, 1, 8, 6, 4), (4, 2, 9, 5, 6), (2, 2, 16, 16, 0), (5, 5, 12, 3, 12), (2, 1, 64, 32, 20)])
def test_qk_prepare_kernel(norm, heads, kv_heads, dim, vdim, rot):
    """Norm, halves rotation and cache store in one launch: every norm with and without weights, both dtypes, a column view of wider
    rows, a token without a slot."""
    from logssms_b200.ops import kernels as K
    T = 7
    g = torch.Generator().manual_seed(dim)
    nq, nk, nv = heads * dim, kv_heads * dim, kv_heads * vdim
    for dtype in DTYPES:
        wide = torch.randn(T, nq + nk + nv + 6, generator=g).to(dtype).cuda()
        qkv = wide[:, :nq + nk + nv]
        positions = torch.randint(0, 50, (T,), generator=g).int()
        slots = torch.tensor([3, 0, 9, 17, -1, 5, 12], dtype=torch.int32)
        a = torch.arange(50, dtype=torch.float64)[:, None] * torch.tensor([7.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float64)
        table = torch.cat([torch.cos(a), torch.sin(a)], 1).float().cuda().contiguous()
        for weighted in (False, True):
            if weighted and norm == "none":
                continue
            wq = (1 + 0.3 * torch.randn(dim if norm == "head" else nq, generator=g)) if weighted else None
            wk = (1 + 0.3 * torch.randn(dim if norm == "head" else nk, generator=g)) if weighted else None
            kc = torch.zeros(2, 10, kv_heads, dim, dtype=dtype, device="cuda")
            vc = torch.zeros(2, 10, kv_heads, vdim, dtype=dtype, device="cuda")
            q = K.qk_prepare(qkv, heads, kv_heads, dim, vdim, positions.cuda(), slots.cuda(), table, norm, None if wq is None else wq.cuda(),
                             None if wk is None else wk.cuda(), EPS, kc, vc)
            x = qkv.double().cpu()
            parts = []
            for rows, H, w in ((x[:, :nq], heads, wq), (x[:, nq:nq + nk], kv_heads, wk)):
                if norm == "row":
                    rows = P.rms(rows, EPS) * (1.0 if w is None else w.double())
                rows = rows.view(T, H, dim)
                if norm == "head":
                    rows = P.rms(rows, EPS) * (1.0 if w is None else w.double())
                parts.append(P.rotate_halves(rows, positions, {"dims": rot, "base": 7.0}) if rot else rows)
            close(q, parts[0], dtype, 1e-5 if dtype == torch.float32 else 1e-2)
            flat_k, flat_v = kc.view(20, kv_heads, dim).cpu(), vc.view(20, kv_heads, vdim).cpu()
            kept = slots >= 0
            close(flat_k[slots[kept].long()], parts[1][kept], dtype, 1e-5 if dtype == torch.float32 else 1e-2)
            assert torch.equal(flat_v[slots[kept].long()], qkv[:, nq + nk:].cpu().view(T, kv_heads, vdim)[kept])
            untouched = [s for s in range(20) if s not in slots.tolist()]
            assert float(flat_k[untouched].abs().sum()) == 0.0


# --------------------------------------------------------------------------- selective scan
def mamba_part(dtype, inner, state, rank, conv, seed=0):
    from logssms_b200.config.specs import MambaSpec
    from logssms_b200.parts import Mamba
    part = Mamba(MambaSpec(WIDTH, inner, state, rank, conv), perturb_init=True)
    return part, give_weights(part, dtype, seed=seed), {"inner": inner, "state": state, "dt_rank": rank}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("inner, state, rank, conv", [(72, 12, 5, 4), (40, 16, 8, 2), (64, 36, 3, 3), (8, 1, 1, 1), (33, 70, 2, 4), (50, 5, 7, 5), (24, 130, 4, 6),
                                                      (16, 200, 2, 1), (136, 8, 16, 4), (7, 3, 9, 8)])
def test_mamba_in_portions(dtype, inner, state, rank, conv):
    part, stored, m = mamba_part(dtype, inner, state, rank, conv, seed=inner + state)
    cache, planner = cache_for([part.cache_needs()], dtype, max_requests=3)
    xs = inputs(LENGTHS, WIDTH, dtype, seed=1)
    for _ in range(2):
        got = step_in_portions(planner, cache, LENGTHS, CUTS, lambda ctx, spans: part.forward(rows_of(xs, spans), ctx, 0))
        for x, y in zip(xs, got):
            close(y, P.mamba(x.double(), f64(stored), m), dtype)


@pytest.mark.parametrize("inner, state, rank, conv", [(40, 16, 4, 4), (24, 7, 3, 3)])
def test_mamba_carries_the_state_through_segments(inner, state, rank, conv):
    """Portions long enough to be cut into segments that run side by side (their edges at multiples of 128 tokens), a portion
    that ends a token behind an edge, beside a short request, and decoded tokens after them; some channels hardly decay."""
    from logssms_b200.ops import kernels as K
    for dtype in DTYPES:
        part, stored, m = mamba_part(dtype, inner, state, rank, conv, seed=state)
        stored["A_log"][::2] = -7.0
        rebind(part, stored, dtype)
        cache, planner = cache_for([part.cache_needs()], dtype, max_requests=3, max_seq_len=1600)
        lengths = [1500, 9, 530]
        assert K.selective_segmented_pays(900, 1, inner, state)
        xs = inputs(lengths, WIDTH, dtype, seed=2)
        got = step_in_portions(planner, cache, lengths, [[900, 2, 0], [513, 1, 520], [1, 1, 1], [84, 5, 2], [1, 0, 1], [1, 0, 6]],
                               lambda ctx, spans: part.forward(rows_of(xs, spans), ctx, 0))
        for x, y in zip(xs, got):
            close(y, P.mamba(x.double(), f64(stored), m), dtype)


def test_mamba_remembers_a_token_hundreds_of_steps_back():
    dtype = torch.float32
    part, stored, m = mamba_part(dtype, 16, 8, 2, 3, seed=4)
    stored["A_log"] = torch.full_like(stored["A_log"], -9.0)
    stored["D"] = torch.zeros_like(stored["D"])
    rebind(part, stored, dtype)
    x = inputs([640], WIDTH, dtype, seed=3)[0] * 0.3
    x[5] *= 40.0
    cache, planner = cache_for([part.cache_needs()], dtype, max_requests=2, max_seq_len=1024)
    cuts = [[300], [1], [1], [2], [250]] + [[1]] * 86
    (got,) = step_in_portions(planner, cache, [640], cuts, lambda ctx, spans: part.forward(rows_of([x], spans), ctx, 0))
    want = P.mamba(x.double(), f64(stored), m)
    close(got, want, dtype)
    blind = x.clone()
    blind[5] = 0.0
    other = P.mamba(blind.double(), f64(stored), m)
    assert float((want - other)[-50:].abs().max() / want[-50:].abs().max()) > 0.05


@pytest.mark.parametrize("inner, n, rank", [(40, 16, 4), (33, 24, 3), (9, 70, 1), (130, 3, 6), (8, 256, 2)])
def test_selective_scan_kernels_equal_the_recurrence(inner, n, rank):
    """The kernels alone, on column views: two portions side by side, the second going on from a state it is handed in another
    slot; with the step's projection handed in, made in the kernel, and (long enough) in segments."""
    from logssms_b200.ops import kernels as K
    from logssms_b200.parts.context import segment_lists
    g = torch.Generator().manual_seed(inner + n)
    lens = [300, 600]
    T = sum(lens)
    xz = torch.randn(T, 2 * inner, generator=g)
    low = torch.randn(T, rank + 2 * n, generator=g)
    dt_w, dt_b = torch.randn(inner, rank, generator=g) * 0.5, torch.randn(inner, generator=g) - 2.0
    A_log, D = torch.randn(inner, n, generator=g), torch.randn(inner, generator=g)
    handed = torch.randn(inner, n, generator=g)
    w = low[:, :rank] @ dt_w.T
    dt = torch.nn.functional.softplus(w.double() + dt_b.double())
    want, states = [], []
    for lo, hi, S0 in ((0, 300, torch.zeros(inner, n)), (300, T, handed)):
        S, A = S0.double(), -torch.exp(A_log.double())
        for t in range(lo, hi):
            S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * xz[t, :inner].double())[:, None] * low[t, rank:rank + n].double()[None]
            want.append((S @ low[t, rank + n:].double() + D.double() * xz[t, :inner].double()) * P.silu(xz[t, inner:].double()))
        states.append(S)
    want = torch.stack(want)
    xz, low = xz.cuda(), low.cuda()
    common = (dt_b.cuda(), A_log.cuda(), D.cuda(), xz[:, inner:])
    where = (i32(0, 300, T), i32(0, 77), i32(0, 2))
    for form in ("handed in", "made", "segments"):
        state = torch.full((3, inner, n), float("nan"))
        state[2] = handed
        state = state.cuda()
        if form == "segments":
            y = torch.empty(T, inner, device="cuda")
            segments, _ = segment_lists(lens, K.SELECTIVE_CHUNK, K.SELECTIVE_SEGMENT, cap_segments=10, cap_long=2)
            K.selective_scan_segments(xz[:, :inner], w.cuda().contiguous(), low, *common, state, *where, torch.from_numpy(segments).cuda(), rank, y)
        else:
            y = K.selective_scan(xz[:, :inner], w.cuda().contiguous() if form == "handed in" else None, low, dt_w.cuda().contiguous(), *common, state,
                                 *where, 2, rank)
        close(y, want, torch.float32, 5e-5)
        close(state[0], states[0], torch.float32, 5e-5)
        close(state[2], states[1], torch.float32, 5e-5)
        assert torch.isnan(state[1]).all()


# --------------------------------------------------------------------------- HGRN2
def hgrn2_part(dtype, heads, dim, vdim, seed=0):
    from logssms_b200.config.specs import HGRN2Spec
    from logssms_b200.parts import HGRN2
    part = HGRN2(HGRN2Spec(WIDTH, heads, dim, vdim, EPS), perturb_init=True)
    return part, give_weights(part, dtype, seed=seed), {"heads": heads, "dim": dim, "vdim": vdim}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dim, vdim", [(3, 16, 24), (2, 32, 40), (1, 1, 2), (4, 8, 16), (2, 48, 72), (3, 20, 5), (1, 128, 32), (2, 160, 8), (1, 260, 12), (2, 64, 64)])
def test_hgrn2_in_portions(dtype, heads, dim, vdim):
    part, stored, m = hgrn2_part(dtype, heads, dim, vdim, seed=heads + dim)
    cache, planner = cache_for([part.cache_needs()], dtype, max_requests=3)
    xs = inputs(LENGTHS, WIDTH, dtype, seed=1)
    for _ in range(2):
        got = step_in_portions(planner, cache, LENGTHS, CUTS, lambda ctx, spans: part.forward(rows_of(xs, spans), ctx, 0))
        for x, y in zip(xs, got):
            close(y, P.hgrn2(x.double(), f64(stored), m, EPS), dtype)


@pytest.mark.parametrize("heads, dim, vdim", [(1, 16, 24), (2, 48, 8), (1, 256, 40)])
def test_hgrn2_carries_the_state_through_segments(heads, dim, vdim):
    """Long portions (segments of 256 tokens side by side in a bfloat16 engine) beside a short request, then decoded tokens; gates
    from hardly open to next to 1, lower bounds of 0 among them."""
    for dtype in DTYPES:
        part, stored, m = hgrn2_part(dtype, heads, dim, vdim, seed=dim)
        stored["f.b"][::3] = 9.0
        stored["f.b"][1::3] = -9.0
        stored["lower"][::2] = 0.0
        rebind(part, stored, dtype)
        cache, planner = cache_for([part.cache_needs()], dtype, max_requests=3, max_seq_len=1600)
        lengths = [1100, 9, 530]
        xs = inputs(lengths, WIDTH, dtype, seed=2)
        got = step_in_portions(planner, cache, lengths, [[600, 2, 0], [413, 1, 520], [1, 1, 1], [84, 5, 2], [1, 0, 1], [1, 0, 6]],
                               lambda ctx, spans: part.forward(rows_of(xs, spans), ctx, 0))
        for x, y in zip(xs, got):
            close(y, P.hgrn2(x.double(), f64(stored), m, EPS), dtype)


def test_hgrn2_remembers_a_token_hundreds_of_steps_back():
    """Gates of 1 but for one token: what it wrote is read unchanged 600 tokens later."""
    dtype = torch.float32
    part, stored, m = hgrn2_part(dtype, 2, 16, 8, seed=4)
    stored["f"] = torch.zeros_like(stored["f"])
    stored["f"][:, 0] = -1.0                                   # the gate follows input column 0
    stored["f.b"] = torch.zeros_like(stored["f.b"])
    rebind(part, stored, dtype)
    x = inputs([640], WIDTH, dtype, seed=3)[0]
    x[:, 0] = -12.0                                            # f = 1 - (1 - l) 6e-6
    x[5, 0] = 3.0
    cache, planner = cache_for([part.cache_needs()], dtype, max_requests=2, max_seq_len=1024)
    cuts = [[300], [1], [1], [2], [250]] + [[1]] * 86
    (got,) = step_in_portions(planner, cache, [640], cuts, lambda ctx, spans: part.forward(rows_of([x], spans), ctx, 0))
    want = P.hgrn2(x.double(), f64(stored), m, EPS)
    close(got, want, dtype)
    blind = x.clone()
    blind[5, 0] = -12.0
    other = P.hgrn2(blind.double(), f64(stored), m, EPS)
    assert float((want - other)[-50:].abs().max() / want[-50:].abs().max()) > 0.05


@pytest.mark.parametrize("H, dk, dv", [(2, 16, 24), (1, 64, 40), (2, 112, 9), (1, 256, 32)])
def test_bounded_gate_chunks_are_sharper_than_bfloat16(H, dk, dv):
    """The chunked kernel hands gates, keys and state to the tensor cores as two bfloat16 terms each: its outputs and states agree
    with the recurrence in float64 (from the same bfloat16 q and v) far closer than 8 bits of mantissa would."""
    from logssms_b200.ops import kernels as K
    from logssms_b200.parts.context import chunk_lists
    g = torch.Generator().manual_seed(dk)
    lens = [70, 41]
    T = sum(lens)
    qv = torch.randn(T, H * (dk + dv), generator=g).bfloat16()
    z, bias = torch.randn(T, H * dk, generator=g) * 3.0, torch.randn(H * dk, generator=g) * 2.0
    lower = torch.rand(H * dk, generator=g) * 0.9
    lower[::4] = 0.0
    z[:, 2::5] = -90.0                                          # gates at their lower bound: at 0 they forget everything
    handed = torch.randn(H, dk, dv, generator=g)
    f = (lower + (1 - lower) * torch.sigmoid((z + bias).double())).view(T, H, dk)
    q, v = P.silu(qv[:, :H * dk].double()).view(T, H, dk), qv[:, H * dk:].double().view(T, H, dv)
    want, states = [], []
    for lo, hi, S0 in ((0, 70, torch.zeros(H, dk, dv)), (70, T, handed)):
        S = S0.double()
        for t in range(lo, hi):
            S = f[t][:, :, None] * S + (1 - f[t])[:, :, None] * v[t][:, None, :]
            want.append((q[t][:, :, None] * S).sum(1).reshape(-1))
        states.append(S)
    want = torch.stack(want)
    chunks, per_request = chunk_lists(lens, K.GLA_CHUNK)
    gate = {"lower": lower.cuda(), "z_bias": bias.cuda()}
    for kernel in ("chunked", "scan"):
        state = torch.full((3, H, dk, dv), float("nan"))
        state[2] = handed
        state = state.cuda()
        where = (i32(0, 70, T), i32(0, 50), i32(0, 2))
        if kernel == "chunked":
            o = torch.empty(T, H * dv, device="cuda")
            K.gla_chunked(qv.cuda(), z.cuda(), state, *where, torch.from_numpy(chunks).cuda(), chunks.shape[0], torch.from_numpy(per_request).cuda(),
                          per_request.shape[0], H, dk, dv, 1.0, 1.0, out=o, **gate)
        else:
            o = K.gla_scan(qv.cuda(), z.cuda(), state, *where, 2, H, dk, dv, 1.0, 1.0, **gate)
        close(o, want, torch.float32, 5e-5)
        close(state[0], states[0], torch.float32, 5e-5)
        close(state[2], states[1], torch.float32, 5e-5)


# --------------------------------------------------------------------------- router and experts
@pytest.mark.parametrize("experts, top, groups, keep", [(12, 4, 3, 2), (16, 5, 8, 4), (6, 6, 2, 2), (9, 4, 3, 2), (4, 1, 4, 1), (1, 1, 1, 1), (64, 8, 4, 2), (250, 7, 1, 1)])
def test_router_with_pairs_of_a_group_and_normalized_weights(experts, top, groups, keep):
    from logssms_b200.ops import kernels as K
    g = torch.Generator().manual_seed(experts)
    T, width = {12: (33, 48), 16: (603, 48), 6: (595, 45)}.get(experts, (33, 51))      # from 592 tokens on a CTA takes four of them
    h, W = torch.randn(T, width, generator=g), torch.randn(experts + 1, width, generator=g) * 0.3
    for shift in (0.0, -2.0):                                  # all choice scores negative the second time
        corr = torch.randn(experts, generator=g) * 0.3 + shift
        dense, chosen, chosen_w, _ = K.moe_route(h.cuda(), W.cuda(), corr.cuda(), experts, top, groups, keep, 1.0, sigmoid_scores=True,
                                                 pair_groups=True, normalize=True, gates=1)
        z = h.double() @ W.double().T
        want = P.route(z[:, :experts], corr.double(), top, groups, keep)
        close(dense[:, :experts], want, torch.float32, 1e-5)
        close(dense[:, experts:], torch.sigmoid(z[:, experts:]), torch.float32, 1e-5)
        assert int((dense[:, :experts] > 0).sum(1).max()) <= top and torch.allclose(chosen_w.sum(1).cpu(), torch.ones(T), atol=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts, top, count, keep, ff, shared", [(12, 3, 4, 2, 16, 24), (6, 2, 3, 2, 22, 14), (1, 1, 1, 1, 8, 1), (10, 5, 5, 3, 7, 9), (8, 2, 2, 1, 32, 40),
                                                                  (4, 2, 2, 2, 12, 0)])
def test_routed_feed_forward(dtype, experts, top, count, keep, ff, shared):
    from logssms_b200.config.specs import RoutedMLPSpec
    from logssms_b200.parts import RoutedMLP
    spec = RoutedMLPSpec(hidden_size=WIDTH, expert_size=ff, num_experts=experts, num_identity=0, top=top, num_groups=count, keep_groups=keep,
                         route_scale=1.0, limit=0.0, score="sigmoid", expert="silu", weigh="output", correction=True, shared_size=shared,
                         shared_gate=shared > 0, group_score="pair", normalize=True)
    part = RoutedMLP(spec)
    stored = give_weights(part, dtype, seed=experts)
    m = {"router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}, "shared": {"ff": shared} if shared else None}
    for n in (1, 5, 90):
        (x,) = inputs([n], WIDTH, dtype, seed=n)
        close(part.forward(x.cuda()), P.moe(x.double(), f64(stored), m), dtype)


# --------------------------------------------------------------------------- input convolution, block, stream
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width, taps", [(56, 4), (24, 1), (64, 2), (31, 3), (40, 8), (16, 5)])
def test_closing_kernel_with_the_next_blocks_convolution(dtype, width, taps):
    """A decode step's closing kernel: addends with a scalar each, the norm, and the convolution from the slots' saved rows, against
    the same in three steps; a request at position 0 starts from zeros whatever its slot holds."""
    from logssms_b200.ops import kernels as K
    g = torch.Generator().manual_seed(width)
    B = 5
    x = torch.randn(B, width, generator=g)
    ys = [torch.randn(B, width, generator=g).to(dtype) for _ in range(3)]
    scales = (0.7, -1.3, 16.0)
    w, cw = torch.full((width,), 0.8), torch.randn(width, taps, generator=g)
    slots, starts = [4, 0, 5, 2, 1], [3, 0, 9, 1, 0]
    state = torch.randn(6, width, max(taps - 1, 1), generator=g).to(dtype)
    state[0] = state[1] = float("nan")
    new = x.double() + sum(s * y.double() for s, y in zip(scales, ys))
    u = (P.rms(new, EPS) * 0.8).to(dtype).double()
    want, after = torch.zeros_like(u), state.clone()
    for b in range(B):
        past = torch.zeros(width, taps - 1, dtype=torch.float64) if starts[b] == 0 else state[slots[b]].double()[:, :taps - 1]
        line = torch.cat([past, u[b][:, None]], 1)
        want[b] = (line * cw.double()).sum(1)
        if taps > 1:
            after[slots[b]] = line[:, 1:].to(dtype)
    xs = x.cuda()
    dev_state = state.cuda() if taps > 1 else None
    h = K.stream_add_conv_step(xs, [(y.cuda(), s) for y, s in zip(ys, scales)], w.cuda(), EPS, "rmsnorm", cw.cuda(), dev_state, i32(*slots), i32(*starts), dtype)
    close(xs, new, torch.float32, 1e-6)
    close(h, want, dtype, 1e-5 if dtype == torch.float32 else 2e-2)
    if taps > 1:
        kept = [4, 0, 5, 2, 1]
        close(dev_state[kept], after[kept], dtype, 1e-5 if dtype == torch.float32 else 1e-2)
        assert torch.equal(dev_state[3].cpu(), state[3])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps, mixer, ff", [(3, "pair", True), (4, "hgrn2", True), (2, "pair", False), (1, "hgrn2", False)])
def test_block_in_portions(dtype, taps, mixer, ff):
    """The block with its input convolution, a mixer of one or two branches, with and without a feed-forward, on a 32-bit stream."""
    from logssms_b200.config import make_model_config
    from logssms_b200.ops import kernels as K
    from logssms_b200.parts import PreNormStreamBlock
    from tiny_dimudra import _hgrn2, _left, _model, _moe, _parallel, _right
    layer = _hgrn2(2, 16, 24) if mixer == "hgrn2" else _parallel(_left(4, 2, 16, 8, 21, 0.4), _right(40, 12, 5, 4), 1.2, 0.7)
    raw = _model(WIDTH, 50, EPS, 1.0, taps, (0, 1, 1), [{**layer, "mlp": _moe(6, 2, 3, 2, 16, 8) if ff else None}])
    block = PreNormStreamBlock(make_model_config(raw).model_spec().layers[0], perturb_init=True)
    stored = give_weights(block, dtype, seed=taps)
    if dtype == torch.bfloat16:
        calm_routers(stored)
        rebind(block, stored, dtype)
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
            want = want + P.mixer(layer["type"], P.input_conv(P.rms(want, EPS) * w["norm1"], w["canon1"]), part("mix."), layer["mixer"], EPS)
            if ff:
                want = want + P.moe(P.rms(want, EPS) * w["norm2"], part("mlp."), raw["layers"][0]["mlp"])
            close(y, want, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_stream_after_every_layer_run(tmp_path, dtype):
    """The stream after every run of every layer (a looped layer once per pass, before the embedding's output is added again), which
    the engine shows to `layer_tap`, and the same logits with and without the tap (the sum then joins in a closing kernel)."""
    from logssms_b200.engine import Engine, StepEntry
    from tiny_dimudra import DIMU_A, make_dimudra_dir, read_folder
    folder = make_dimudra_dir(tmp_path / "m", DIMU_A, seed=3, dtype=torch.float32 if dtype == "float32" else torch.bfloat16, calm=dtype == "bfloat16")
    ids = [int(i) for i in torch.randint(0, 211, (37,), generator=torch.Generator().manual_seed(2))]
    config, tensors = read_folder(folder)
    logits, streams = P.forward(config, tensors, ids, want_layers=True)
    engine = Engine(folder, dtype, max_requests=2, max_seq_len=64, num_pages=2, use_graphs=False)
    seen = []
    engine.layer_tap = lambda i, x, residual: seen.append(x.f32.clone())
    r = engine.new_request()
    a = engine.step([StepEntry(r, ids, list(range(len(ids))))]).clone()
    engine.release(r)
    assert len(seen) == streams.shape[0] == 8
    tol = 2e-5 if dtype == "float32" else 6e-2
    for i, s in enumerate(seen):
        err = (s.double().cpu() - streams[i]).pow(2).mean().sqrt() / streams[i].pow(2).mean().sqrt()
        assert float(err) < tol, (i, float(err))
    engine.layer_tap = None
    r = engine.new_request()
    b = engine.step([StepEntry(r, ids, list(range(len(ids))))])
    close(b, a, torch.float32, 1e-5 if dtype == "float32" else 1e-2)
    if dtype == "float32":
        close(a, logits, torch.float32, 1e-4)
