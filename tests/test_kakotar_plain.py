"""What needs no GPU of the Kakotar design: its configuration and plan, the plain
implementation's reading of each mechanism against hand computation, and the cache's
bookkeeping for chunks and for windows that another layer reads through."""
import json
import math

import pytest
import torch

from plain import kakotar as plain

ROT = {"base": 100.0, "dims": 4}
CFG = dict(architecture="Kakotar", vocab=50, width=16, norm={"eps": 1e-5}, layers=[
    dict(type="attention", mixer=dict(heads=2, kv_heads=1, dim=8, vdim=4, scale=0.3, mask={"size": 3},
                                      rot=dict(ROT, scaling={"factor": 2.0, "original": 64, "fast": 8.0, "slow": 1.0})),
         mlp={"kind": "moe", "expert": {"ff": 8}, "shared": {"ff": 12},
              "router": {"experts": 6, "top": 2, "scale": 2.0, "groups": {"count": 3, "keep": 2}}}),
    dict(type="lightning", mixer=dict(heads=3, dim=4, vdim=6, decay=[0.5, 0.9, 1.0]), mlp=None),
    dict(type="attention", mixer=dict(heads=4, kv_heads=1, dim=8, vdim=4, scale=0.2, mask={"size": 90}, kv_from=0,
                                      rot=dict(ROT, scaling={"factor": 2.0, "original": 64, "fast": 8.0, "slow": 1.0})),
         mlp=None),
    dict(type="attention_2", mixer=dict(heads=2, kv_heads=2, dim=6, vdim=10, scale=0.5, diff=0.4, mask={"size": 5},
                                        rot={"base": 50.0, "dims": 2, "scaling":
                                             {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 32}}),
         mlp={"kind": "moe", "expert": {"ff": 4}, "router": {"experts": 1, "top": 1, "scale": 1.0}})])


def _plan(cfg):
    import grout_b200.architectures  # noqa: F401
    from grout_b200.config import resolve_architecture
    arch = resolve_architecture(cfg)
    return arch.plan(arch.config_cls.from_dict(cfg))


def test_configuration_names_every_problem():
    import grout_b200.architectures  # noqa: F401
    from grout_b200.config import ConfigError, KakotarConfig, resolve_architecture
    assert resolve_architecture(CFG).name == "Kakotar"
    KakotarConfig.from_dict(CFG)
    bad = json.loads(json.dumps(CFG))
    L = bad["layers"]
    L[0]["mixer"]["rot"]["dims"] = 10                       # more than a head has
    L[0]["mixer"]["rot"]["scaling"] = {"factor": 2.0, "original": 64, "fast": 8.0}
    L[0]["mlp"]["router"]["groups"]["count"] = 4            # six experts do not form four groups
    L[1]["mixer"]["decay"] = [0.5, 0.9]                     # three heads
    L[2]["mixer"]["kv_heads"] = 2                           # not those of the layer it reads
    L[3]["mixer"]["mask"] = {"size": 0}
    del L[3]["mixer"]["diff"]
    del L[3]["mlp"]["router"]["scale"]
    del bad["norm"]["eps"]
    with pytest.raises(ConfigError) as e:
        KakotarConfig.from_dict(bad)
    assert len(e.value.problems) == 9, e.value.problems
    for src, words in ((1, "type 'attention'"), (2, "earlier"), (3, "earlier"), (-1, "earlier")):
        bad = json.loads(json.dumps(CFG))
        bad["layers"][2]["mixer"]["kv_from"] = src
        with pytest.raises(ConfigError) as e:
            KakotarConfig.from_dict(bad)
        assert len(e.value.problems) == 1 and words in e.value.problems[0], e.value.problems
    bad = json.loads(json.dumps(CFG))
    bad["layers"][0]["type"] = "window"
    bad["layers"][3]["mlp"]["kind"] = "dense"
    with pytest.raises(ConfigError) as e:
        KakotarConfig.from_dict(bad)
    assert len(e.value.problems) == 3, e.value.problems      # (and layer 2 no longer reads an attention layer)


def test_plan_reads_exactly_the_designs_tensors():
    from grout_b200.engine.model import expected_tensors
    exp = expected_tensors(_plan(CFG))
    shapes = {n: tuple(s.shape) for n, s in exp.items()}
    assert shapes["embed"] == shapes["head"] == (50, 16)
    assert shapes["final.norm"] == shapes["final.norm.b"] == (16,) and shapes["final.norm.alpha"] == ()
    assert shapes["l0.norm1"] == (16,) and shapes["l0.norm2.alpha"] == () and "l1.norm2" not in shapes
    assert shapes["l0.mix.q"] == (16, 16) and shapes["l0.mix.k"] == (8, 16) and shapes["l0.mix.v"] == (4, 16)
    assert shapes["l0.mix.o"] == (16, 8)
    assert shapes["l0.mlp.e5.up"] == (8, 16) and shapes["l0.mlp.e5.down"] == (16, 8) and "l0.mlp.e0.gate" not in shapes
    assert shapes["l0.mlp.correction"] == (6,) and shapes["l0.mlp.shared.up"] == (12, 16)
    assert shapes["l1.mix.v"] == shapes["l1.mix.g"] == (18, 16) and shapes["l1.mix.norm"] == (18,)
    assert shapes["l2.mix.q"] == (32, 16) and shapes["l2.mix.o"] == (16, 16)
    assert "l2.mix.k" not in shapes and "l2.mix.v" not in shapes
    assert shapes["l3.mix.q"] == (24, 16) and shapes["l3.mix.k"] == (24, 16) and shapes["l3.mix.v"] == (20, 16)
    assert shapes["l3.mix.lq2"] == (6,) and shapes["l3.mix.o"] == (16, 20)
    assert shapes["l3.mlp.correction"] == (1,) and "l3.mlp.shared.up" not in shapes


def test_needs_of_the_cache_and_a_readers_longer_window():
    from grout_b200.cache import KVSpec, StateSpec
    from grout_b200.engine.model import Model
    from grout_b200.parts import BuildContext
    model = Model(_plan(CFG), BuildContext(torch.float32, torch.device("cpu")))
    specs = [b.cache_spec() for b in model.blocks]
    assert specs[0] == KVSpec(1, 8, 90)          # its own window is 3, its reader's 90
    assert specs[1] == StateSpec((3 * 4 * 6,)) and specs[2] is None
    assert specs[3] == KVSpec(2, 12, None, chunk=5)
    assert [e.cache_of for e in model.plan.schedule] == [None, None, 0, None]
    assert model.blocks[0].mixer.window == 3 and model.blocks[2].mixer.window == 90
    for readers, kept in ((None, 3), ({"size": 2}, 3), ("absent", None)):
        cfg = json.loads(json.dumps(CFG))
        if readers is None:
            del cfg["layers"][2]
        elif readers == "absent":
            del cfg["layers"][2]["mixer"]["mask"]
        else:
            cfg["layers"][2]["mixer"]["mask"] = readers
        model = Model(_plan(cfg), BuildContext(torch.float32, torch.device("cpu")))
        assert model.blocks[0].cache_spec().window == kept
    half = Model(_plan(CFG), BuildContext(torch.bfloat16, torch.device("cpu")))
    assert [b.cache_spec().head_dim for b in (half.blocks[0], half.blocks[3])] == [16, 16]    # rows of whole sixteens


def test_a_chunked_store_gives_back_what_lies_in_front_of_the_next_tokens_chunk():
    from grout_b200.cache import CacheLayout, KVSpec, SequenceCache
    cache = SequenceCache(CacheLayout.from_specs([KVSpec(1, 8, None, chunk=100), KVSpec(1, 8, 100), KVSpec(1, 8)]),
                          max_tokens=64 * 40, max_slots=4, max_seq_len=2048, dtype=torch.float32, device="cpu",
                          allocate=False)
    s = cache.open()
    for n, first in ((64, 0), (35, 0), (1, 1), (100, 3), (99, 3), (1, 4), (300, 9)):
        cache.reserve(s, n)
        cache.advance(s, n)
        cache.check()
        pages, length = cache.stores[0].pages_of[s], cache.length[s]
        # the next token's chunk begins at length // 100 * 100: pages wholly in front of it are free
        assert first == length // 100 * 100 // 64
        assert all(p is None for p in pages[:first]) and all(p is not None for p in pages[first:]), length
    assert [st.tokens_held() // 64 for st in cache.stores] == [1, 3, 10]      # 600 tokens
    other = cache.open()
    cache.reserve(other, 130)
    cache.close(s)
    cache.check()
    assert [st.tokens_held() // 64 for st in cache.stores] == [3, 3, 3]
    cache.close(other)
    assert cache.tokens_held() == 0


def test_masks_by_hand():
    w, c = plain.window_mask(8, 3), plain.chunk_mask(8, 3)
    assert w[5].tolist() == [False, False, False, True, True, True, False, False]
    assert c[5].tolist() == [False, False, False, True, True, True, False, False]
    assert c[6].tolist() == [False] * 6 + [True, False] and c[7].tolist() == [False] * 6 + [True, True]
    assert c[2].tolist() == [True] * 3 + [False] * 5 and plain.window_mask(4, 1).equal(torch.eye(4, dtype=torch.bool))


def test_frequencies_by_hand():
    base, dims = 1e4, 16
    f = plain.plain_frequencies(base, dims)
    assert f[0] == 1.0 and abs(f[4] - 0.01) < 1e-15
    # turns within 1000 positions: element e(t) = 16 ln(1000 / (2 pi t)) / (2 ln 1e4)
    e = lambda t: 16 * math.log(1000 / (2 * math.pi * t)) / (2 * math.log(1e4))
    lo, hi = math.floor(e(32.0)), math.ceil(e(1.0))
    assert (lo, hi) == (1, 5)
    y = plain.yarn_frequencies(base, dims, 4.0, 1000, 32.0, 1.0)
    assert y[:2] == f[:2] and all(abs(y[i] - f[i] / 4) < 1e-18 for i in (5, 6, 7))
    assert abs(y[3] - (f[3] / 4 * 0.5 + f[3] * 0.5)) < 1e-15          # half way up the ramp
    assert plain.yarn_amplitude(1.0) == 1.0 and abs(plain.yarn_amplitude(math.e) - 1.1) < 1e-15
    b = plain.banded_frequencies(base, dims, 8.0, 1.0, 4.0, 64)
    wave = [2 * math.pi / x for x in f]
    assert b[0] == f[0] and wave[0] < 16 and b[7] == f[7] / 8 and wave[7] > 64
    i = next(j for j in range(8) if 16 < wave[j] < 64)
    s = (64 / wave[i] - 1.0) / 3.0
    assert abs(b[i] - ((1 - s) * f[i] / 8 + s * f[i])) < 1e-15
    from grout_b200.parts.position import scaled_inverse_frequencies
    got = scaled_inverse_frequencies(dims, base, {"factor": 4.0, "original": 1000, "fast": 32.0, "slow": 1.0})
    assert all(abs(g - y_i) <= 1e-15 * y_i for g, y_i in zip(got, y))


def test_rotation_and_amplitude_by_hand():
    x = torch.tensor([[1.0, 2.0, 3.0, 4.0, 5.0]])
    y = plain.rotate(x, [2], [0.5, 0.1], 1.5)[0]
    c, s = math.cos(1.0), math.sin(1.0)
    assert abs(float(y[0]) - 1.5 * (c - 3 * s)) < 1e-12 and abs(float(y[2]) - 1.5 * (3 * c + s)) < 1e-12
    assert abs(float(y[1]) - 1.5 * (2 * math.cos(0.2) - 4 * math.sin(0.2))) < 1e-12 and float(y[4]) == 5.0


def test_difference_factor_and_differential_attention_of_one_token():
    m = dict(heads=1, kv_heads=1, dim=2, vdim=3, scale=1.0, diff=0.25)
    w = {"q": torch.zeros(4, 3), "k": torch.zeros(4, 3), "v": torch.eye(3), "o": torch.eye(3),
         "lq1": torch.tensor([1.0, 2.0]), "lk1": torch.tensor([0.5, 0.25]), "lq2": torch.tensor([1.0, 0.0]),
         "lk2": torch.tensor([0.0, 3.0])}
    w = {"m." + k: v for k, v in w.items()}
    lam = plain.difference_factor(w, "m.", 0.25)
    assert abs(lam - (math.exp(1.0) - 1.0 + 0.25)) < 1e-12
    h = torch.tensor([[3.0, 0.0, 4.0]], dtype=torch.float64)
    y = plain.differential_attention(h, w, "m.", m, [0], 0.0)[0]     # one key: both maps are v
    o = (1 - lam) * h[0]
    assert torch.allclose(y, o / math.sqrt(float((o * o).mean())) * 0.75)


def test_fading_state_by_hand():
    one = lambda *v: torch.tensor(v).view(-1, 1)
    o, S = plain.fading_state_head(one(1.0, 1.0, 2.0), one(1.0, 0.0, 3.0), one(4.0, 9.0, 1.0), 0.5)
    assert o.view(-1).tolist() == [4.0, 2.0, 8.0] and float(S) == 4.0


def test_choice_and_weights_by_hand():
    s = torch.tensor([0.9, 0.1, 0.6, 0.5, 0.2, 0.3], dtype=torch.float64)
    r = {"top": 2, "scale": 3.0, "groups": {"count": 3, "keep": 1}}
    chosen, w = plain.route(s, torch.zeros(6), r)             # 1.0, 1.1 and 0.5: the second group
    assert chosen == [2, 3] and torch.allclose(w, torch.tensor([0.6, 0.5], dtype=torch.float64) / 1.1 * 3)
    chosen, w = plain.route(s, torch.tensor([-5.0, -5, -5, -5, -1.2, -1.0]), r)
    assert chosen == [5, 4] and torch.allclose(w, torch.tensor([0.3, 0.2], dtype=torch.float64) / 0.5 * 3)
    chosen, _w = plain.route(s, torch.zeros(6), dict(r, groups=None))
    assert chosen == [0, 2]


def test_the_models_norm_looks_at_single_elements():
    w = {"n": torch.tensor([2.0, 1.0]), "n.b": torch.tensor([0.0, -1.0]), "n.alpha": torch.tensor(0.5)}
    y = plain.dynamic_tanh(torch.tensor([[1.0, 50.0]]), w, "n")[0]
    assert abs(float(y[0]) - 2 * math.tanh(0.5)) < 1e-12 and abs(float(y[1])) < 1e-12
