"""Fosupel on the CPU: configuration and its refusals, tensor names, the looped schedule, cache needs, pages of kept first tokens,
rotation frequencies, and the plain functions against cases worked out by hand."""
import copy
import math
import random

import pytest
import torch

from logssms_b200.cache import CacheManager, CacheNeeds, KVNeed, OutOfPages, PagedNeed, PagedTensor
from logssms_b200.config import ConfigError, make_model_config
from logssms_b200.models import build_model
from plain import fosupel_plain as P
from tiny_fosupel import FOSU, FOSU_A, FOSU_B, FOSU_C, FOSU_D, FOSU_E

D = torch.float64


# --------------------------------------------------------------------------- configuration
def test_config_round_trip_and_specs():
    cfg = make_model_config(FOSU_A)
    assert cfg.to_dict() == FOSU_A and cfg.architectures == ("Fosupel",)
    spec = cfg.model_spec()
    assert [b.mixer.spec.kind for b in spec.layers] == ["mixer_pair", "latent_attention", "mixer_pair", "latent_attention"]
    assert [None if b.feed_forward is None else b.feed_forward.kind for b in spec.layers] == ["dense_mlp", "routed_mlp", "routed_mlp", None]
    assert all(b.residual_scale == 0.6 and b.kind == "prenorm_stream" for b in spec.layers)
    assert spec.tie_word_embeddings and spec.lm_head_kind == "lm_head_softcap" and dict(spec.lm_head_options) == {"cap": 12.0}
    pair = spec.layers[0].mixer.spec
    a, b = pair.left.spec, pair.right.spec
    assert (pair.left.out_scale, pair.right.out_scale) == (0.8, 1.3)
    assert (a.num_heads, a.num_kv_heads, a.head_dim, a.value_dim, a.window, a.keep_first, a.softmax_scale, a.sink) == (6, 2, 16, 24, 20, 5, 0.3, True)
    assert (a.position.rotary_dim, a.position.theta, dict(a.position.scaling)) == (8, 500.0, {"factor": 3.0})
    assert (b.num_heads, b.key_dim, b.value_dim, b.decay) == (3, 16, 24, (0.75, 1 - 2.0 ** -5, 1 - 2.0 ** -8)) and b.position.scaling is None
    lat = spec.layers[1].mixer.spec
    assert (lat.num_heads, lat.nope_dim, lat.rot_dim, lat.value_dim, lat.kv_rank) == (4, 16, 8, 24, 40)
    assert lat.pairing == "neighbours" and lat.sink and lat.column_gate and not lat.head_gate and lat.window is None
    ff, routed = spec.layers[0].feed_forward, spec.layers[1].feed_forward
    assert (ff.activation, ff.intermediate_size) == ("xielu", 72)
    assert (routed.num_experts, routed.top, routed.expert_size, routed.shared_size, routed.shared_gate) == (6, 2, 24, 8, True)
    assert routed.score == "softmax" and not routed.correction and not routed.normalize and routed.expert == "silu" and routed.num_groups == 1
    no_shared = make_model_config(FOSU_B).model_spec().layers[0].feed_forward
    assert no_shared.shared_size == 0 and not no_shared.shared_gate
    bare = make_model_config(FOSU_C).model_spec()
    assert bare.layers[0].mixer.spec.left.spec.position is None and bare.layers[1].mixer.spec.rot_dim == 0
    open_window = make_model_config(FOSU_D).model_spec().layers[0].mixer.spec.left.spec
    assert open_window.window is None and open_window.keep_first == 0


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="mamba"), "is not a mixer"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(heads=5), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(dim=0), "dim must be positive"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(dim=2000), "at most 1024"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "mask.size must be positive"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(keep_first=-1), "keep_first must not be negative"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "rot.dims must be even"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "at most 16"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(base=0), "rot.base must be positive"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=0), "factor must be positive"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5, 0.5]), "one decay within"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5, 1.5, 0.5]), "one decay within"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(dim=600), "at most 512"),
    (lambda c: c["layers"][1]["mixer"].update(rot_dim=3), "rot_dim must be even"),
    (lambda c: c["layers"][1]["mixer"].update(kv_rank=1000), "at most 512"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), "at most 8"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "router.top"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(experts=300), "at most 256"),
    (lambda c: c["layers"][1]["mlp"]["shared"].update(ff=0), "shared.ff must be positive"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "neither 'dense' nor 'moe'"),
    (lambda c: c["norm"].update(eps=0.0), "norm.eps"),
    (lambda c: c.update(logit_softcap=0), "logit_softcap"),
    (lambda c: c["loop"].update(stop=9), "loop must name"),
    (lambda c: c["loop"].update(times=0), "loop must name"),
])
def test_config_refusals(change, message):
    raw = copy.deepcopy(FOSU_A)
    change(raw)
    with pytest.raises(ConfigError, match=message):
        make_model_config(raw)


@pytest.mark.parametrize("path", [("vocab",), ("width",), ("norm",), ("residual_mult",), ("logit_softcap",), ("layers", 0, "mixer", "left"),
                                  ("layers", 0, "mixer", "right", "vdim"), ("layers", 0, "mixer", "left", "scale"), ("layers", 0, "mixer", "left_scale"),
                                  ("layers", 1, "mixer", "rot_dim"), ("layers", 1, "mlp", "router"), ("layers", 0, "mlp", "ff")])
def test_missing_keys_are_refused(path):
    raw = copy.deepcopy(FOSU_A)
    at = raw
    for key in path[:-1]:
        at = at[key]
    del at[path[-1]]
    with pytest.raises(ConfigError):
        make_model_config(raw)


@pytest.mark.parametrize("raw, runs", [
    (FOSU_A, [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]),
    (FOSU_B, [(0, 0), (1, None), (0, 1), (1, None)]),
    (FOSU_D, [(0, None), (1, None)]),
    (FOSU_E, [(0, None), (1, None), (2, 0), (2, 1), (2, 2), (2, 3), (3, None)]),
])
def test_looped_schedule(raw, runs):
    cfg = make_model_config(raw)
    assert cfg.layer_runs() == runs == P.layer_runs(raw)
    schedule = cfg.model_spec().resolved_schedule()
    assert [(e.layer, e.turn if e.opens is not None else None) for e in schedule] == runs
    assert [e.cache for e in schedule] == list(range(len(runs)))            # every run has a cache layer of its own
    assert len(build_model(cfg).cache_needs()) == len(runs)


def names_of(raw):
    return {n: tuple(s.shape) for n, s in dict(build_model(make_model_config(raw)).named_param_specs()).items()}


def test_tensor_names_and_shapes():
    names = names_of(FOSU_A)
    want = {"embed": (211, 64), "loop.step": (3, 64), "final.norm": (64,), "l0.norm1": (64,), "l0.norm2": (64,),
            "l0.mix.left.q": (96, 64), "l0.mix.left.k": (32, 64), "l0.mix.left.v": (48, 64), "l0.mix.left.talk": (6, 6),
            "l0.mix.left.sink": (6,), "l0.mix.left.o": (64, 144), "l0.mix.right.q": (48, 64), "l0.mix.right.k": (48, 64),
            "l0.mix.right.v": (72, 64), "l0.mix.right.g": (72, 64), "l0.mix.right.o": (64, 72), "l0.mlp.up": (72, 64),
            "l0.mlp.down": (64, 72), "l0.mlp.act": (2,), "l1.mix.q": (96, 64), "l1.mix.dkv": (48, 64), "l1.mix.dkv.norm": (40,),
            "l1.mix.uk": (64, 40), "l1.mix.uv": (96, 40), "l1.mix.sink": (4,), "l1.mix.g": (96, 64), "l1.mix.o": (64, 96),
            "l1.mlp.router": (6, 64), "l1.mlp.e5.gate": (24, 64), "l1.mlp.e5.down": (64, 24), "l1.mlp.shared.up": (8, 64),
            "l1.mlp.shared.sg": (1, 64), "l3.norm1": (64,)}
    for n, shape in want.items():
        assert names[n] == shape, n
    assert not any(n.startswith("l3.norm2") or n.startswith("l3.mlp") or n.startswith("head") or "correction" in n for n in names)
    assert not any("shared" in n for n in names_of(FOSU_B)) and "loop.step" not in names_of(FOSU_D)


# --------------------------------------------------------------------------- cache
def test_cache_needs():
    needs = build_model(make_model_config(FOSU_A)).cache_needs()
    assert needs[0].kv == KVNeed(2, 16, 20, 24, keep_first=5) and [(s.name, s.shape, s.dtype) for s in needs[0].states] == [("retention", (3, 16, 24), torch.float32)]
    assert needs[1].kv == PagedNeed((PagedTensor("c", (40,)), PagedTensor("kr", (8,)))) and not needs[1].states
    with pytest.raises(ValueError, match="keeps its first tokens beside a window"):
        KVNeed(1, 4, None, 4, keep_first=3)


@pytest.mark.parametrize("keep, kept_pages", [(0, 0), (1, 1), (16, 1), (17, 2), (40, 3)])
def test_pages_of_kept_first_tokens_stay(keep, kept_pages):
    m = CacheManager([CacheNeeds(kv=KVNeed(1, 4, 20, 4, keep_first=keep))], page_size=16, num_pages=20, max_requests=2, max_seq_len=320,
                     dtype=torch.float32, device="cpu", poison_on_free=True)
    (g,) = m.groups
    a = m.admit()
    m.extend(a, 7)
    first = int(g.block_table[a.row, 0])
    g.tensor("k", 0)[first] = 1.0
    for n in range(8, 300):
        m.extend(a, n)
        m.check_integrity()
        table = g.block_table[a.row]
        oldest = max(0, n - 1 - 20 + 1) // 16                   # the page of the oldest token the newest one sees in its window
        for p in range(-(-n // 16)):
            assert (table[p] >= 0) == (p < kept_pages or p >= oldest), (n, p)
        assert g.pool.num_held <= kept_pages + 3
    if kept_pages:
        assert int(g.block_table[a.row, 0]) == first and float(g.tensor("k", 0)[first].min()) == 1.0
    b = m.admit()
    m.extend(b, 100)
    m.check_integrity()
    m.release(a)
    m.check_integrity()
    m.release(b)
    assert g.pool.num_held == 0 and torch.isnan(g.tensor("k", 0)[first]).all()


def test_random_growth_and_release_with_kept_tokens():
    rng = random.Random(5)
    needs = [CacheNeeds(kv=KVNeed(1, 4, 24, 4, keep_first=20)), CacheNeeds(kv=KVNeed(1, 4)), CacheNeeds(kv=KVNeed(1, 4, 5, 4, keep_first=3))]
    m = CacheManager(needs, page_size=8, num_pages=26, max_requests=5, max_seq_len=200, dtype=torch.float32, device="cpu", max_step_tokens=30)
    live = []
    for _ in range(1500):
        action = rng.random()
        if action < 0.25 and m.rows.num_free:
            reserve = rng.choice([0, 0, rng.randrange(1, 120)])
            if m.can_admit(reserve):
                live.append((m.admit(reserve), reserve))
        elif action < 0.9 and live:
            rc, reserve = rng.choice(live)
            n = min(reserve if reserve else 200, rc.length + rng.choice([1, 1, 1, 2, 7, 30]))
            fits = True
            try:
                m.check_room([(rc, n)])
            except OutOfPages:
                fits = False
            try:
                m.extend(rc, n)
                assert fits
            except OutOfPages:
                assert reserve == 0 and not fits           # the room check says the same; a reserved request never runs dry
        elif live:
            rc, _ = live.pop(rng.randrange(len(live)))
            m.release(rc)
        m.check_integrity()
    for rc, _ in live:
        m.release(rc)
    m.check_integrity()
    assert all(g.pool.num_held == 0 for g in m.groups)


# --------------------------------------------------------------------------- parts without a GPU
def test_linear_frequencies():
    from logssms_b200.config.specs import RopeSpec
    from logssms_b200.parts import LinearRotaryEmbedding
    f, magnitude = LinearRotaryEmbedding(RopeSpec(16, 8, 500.0, 100, (("factor", 3.0),), kind="rope_linear")).frequencies()
    assert magnitude == 1.0 and torch.allclose(f.double(), torch.tensor([500.0 ** (-i / 4) / 3.0 for i in range(4)], dtype=D), rtol=1e-7)
    f, _ = LinearRotaryEmbedding(RopeSpec(16, 4, 9.0, 100, None, kind="rope_linear")).frequencies()
    assert torch.allclose(f.double(), torch.tensor([1.0, 1 / 3.0], dtype=D), rtol=1e-7)


def test_parts_refuse_what_they_have_no_kernels_for():
    from dataclasses import replace
    from logssms_b200.parts import DenseMLP, LatentAttention, PreNormStreamBlock, TalkingAttention
    spec = make_model_config(FOSU_A).model_spec()
    with pytest.raises(ValueError, match="gelu_tanh and xielu"):
        DenseMLP(replace(spec.layers[0].feed_forward, activation="relu"))
    with pytest.raises(ValueError, match="not both"):
        LatentAttention(replace(spec.layers[1].mixer.spec, head_gate=True))
    with pytest.raises(ValueError, match="kept beside a window"):
        TalkingAttention(replace(spec.layers[0].mixer.spec.left.spec, window=None))
    with pytest.raises(ValueError, match="without layer scales"):
        PreNormStreamBlock(replace(spec.layers[0], layer_scale=True))


# --------------------------------------------------------------------------- the plain functions by hand
def test_plain_mask_keeps_first_tokens():
    seen = P.seen_by(7, {"size": 2, "keep_first": 2})
    assert [[j for j in range(7) if seen[i, j]] for i in range(7)] == [[0], [0, 1], [0, 1, 2], [0, 1, 2, 3], [0, 1, 3, 4], [0, 1, 4, 5], [0, 1, 5, 6]]
    assert torch.equal(P.seen_by(5, None), torch.tril(torch.ones(5, 5)).bool())


def test_plain_talking_attention_by_hand():
    """Two heads of one key/value head, two tokens, scores of zero: head weights 1 / (n + e^sink), mixed by the matrix."""
    v = torch.tensor([[[1.0]], [[10.0]]], dtype=D)
    talk = torch.tensor([[2.0, -1.0], [0.5, 3.0]], dtype=D)
    sink = torch.tensor([0.0, math.log(2.0)], dtype=D)
    o = P.talking_attention(torch.zeros(2, 2, 1, dtype=D), torch.zeros(2, 1, 1, dtype=D), v, 1.0, None, sink, talk)
    for i, total in ((0, 1.0), (1, 11.0)):
        u = [total / (i + 1 + 1), total / (i + 1 + 2)]
        assert torch.allclose(o[i, :, 0], talk @ torch.tensor(u, dtype=D))
    # a second key/value head: every head's weights meet the values of the head that applies them
    v = torch.tensor([[[1.0], [100.0]]], dtype=D)
    o = P.talking_attention(torch.zeros(1, 2, 1, dtype=D), torch.zeros(1, 2, 1, dtype=D), v, 1.0, None, sink, talk)
    mixed = talk @ torch.tensor([1 / 2, 1 / 3], dtype=D)
    assert torch.allclose(o[0, :, 0], mixed * torch.tensor([1.0, 100.0], dtype=D))


def test_plain_memory_and_rotation_by_hand():
    one = torch.ones(3, 1, 1, dtype=D)
    o = P.decayed_memory(one, one, one, torch.tensor([0.5], dtype=D))
    assert o.flatten().tolist() == [1.0, 1.5, 1.75]
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]]], dtype=D)
    pos, rot = torch.tensor([3]), {"dims": 4, "base": 16.0, "scaling": {"factor": 2.0}}
    a, b = 1.5, 3 / 8.0                                        # 3 / 2, 3 * 16^(-1/2) / 2
    want = [math.cos(a) - 3 * math.sin(a), 2 * math.cos(b) - 4 * math.sin(b), 3 * math.cos(a) + math.sin(a), 4 * math.cos(b) + 2 * math.sin(b), 5.0]
    assert torch.allclose(P.rotate_halves(x, pos, rot).flatten(), torch.tensor(want, dtype=D))
    want = [math.cos(a) - 2 * math.sin(a), 2 * math.cos(a) + math.sin(a), 3 * math.cos(b) - 4 * math.sin(b), 4 * math.cos(b) + 3 * math.sin(b), 5.0]
    assert torch.allclose(P.rotate_neighbours(x, pos, rot).flatten(), torch.tensor(want, dtype=D))


def test_plain_xielu_and_router_by_hand():
    p, q = torch.tensor(0.3, dtype=D), torch.tensor(-0.7, dtype=D)
    a, b = math.log1p(math.exp(0.3)), 0.5 + math.log1p(math.exp(-0.7))
    got = P.xielu(torch.tensor([2.0, 0.0, -1.0], dtype=D), p, q)
    assert torch.allclose(got, torch.tensor([4 * a + 1.0, 0.0, b * (math.exp(-1.0) - 1 + 1) - 0.5], dtype=D))
    w = P.route(torch.tensor([[0.0, math.log(2.0), math.log(5.0)]], dtype=D), 2)
    assert torch.allclose(w, torch.tensor([[0.0, 2 / 8, 5 / 8]], dtype=D))


@pytest.mark.parametrize("name", ["A", "C", "E"])
def test_plain_model_is_causal_and_capped(tmp_path, name):
    from tiny_fosupel import make_fosupel_dir, plain_logits
    raw = FOSU[name]
    folder = make_fosupel_dir(tmp_path / "m", raw, seed=1)
    ids = [int(i) for i in torch.randint(0, raw["vocab"], (40,), generator=torch.Generator().manual_seed(0))]
    full = plain_logits(folder, ids)
    assert torch.allclose(plain_logits(folder, ids[:23]), full[:23], atol=1e-9) and float(full.abs().max()) <= raw["logit_softcap"]
