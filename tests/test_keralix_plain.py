"""What needs no GPU of the Keralix design: its configuration and plan, what it asks of the
cache, tensors whose inner size no configuration states, and the plain implementation's
reading of each mechanism against hand computation."""
import json
import math

import pytest
import torch

from plain import keralix as plain

ATT = dict(heads=4, kv_heads=2, dim=6, vdim=6, conv=3, scale=0.3, softcap=20.0, rot={"base": 100.0, "dims": 4}, mask={"size": 5})
LAT = dict(heads=3, dim=8, vdim=4, q_rank=10, kv_rank=12, scale=0.2)
DEL = dict(heads=4, kv_heads=2, dim=8, vdim=6, conv=4)
CFG = dict(architecture="Keralix", vocab=50, width=16, streams=3, norm={"eps": 1e-5}, embedding={"scale": 2.0}, layers=[
    dict(type="attention", mixer=ATT, mlp={"kind": "dense", "ff": 24}),
    dict(type="latent_attention", mixer=LAT, mlp=None),
    dict(type="channel_delta", mixer=DEL, mlp={"kind": "dense", "ff": 40})])


def _plan(cfg):
    import grout_b200.architectures  # noqa: F401
    from grout_b200.config import resolve_architecture
    arch = resolve_architecture(cfg)
    return arch.plan(arch.config_cls.from_dict(cfg))


def test_configuration_names_every_problem():
    import grout_b200.architectures  # noqa: F401
    from grout_b200.config import ConfigError, KeralixConfig, resolve_architecture
    assert resolve_architecture(CFG).name == "Keralix"
    KeralixConfig.from_dict(CFG)
    bad = json.loads(json.dumps(CFG))
    L = bad["layers"]
    L[0]["mixer"].update(vdim=8, rot={"base": 100.0, "dims": 8}, mask={"size": 0}, softcap=-1.0)
    L[1]["mixer"]["q_rank"] = 0
    L[2]["mixer"]["kv_heads"] = 3
    L[2]["mlp"] = {"kind": "moe"}
    bad["streams"] = 17
    del bad["norm"]["eps"]
    with pytest.raises(ConfigError) as e:
        KeralixConfig.from_dict(bad)
    assert len(e.value.problems) == 9, e.value.problems
    for key in ("streams", "embedding", "norm", "layers"):
        with pytest.raises(ConfigError, match=key):
            KeralixConfig.from_dict({k: v for k, v in CFG.items() if k != key})
    # a rotation, a window and a cap may be absent
    plain_att = {k: v for k, v in ATT.items() if k not in ("rot", "mask", "softcap")}
    KeralixConfig.from_dict(dict(CFG, layers=[dict(type="attention", mixer=plain_att, mlp=None)]))


def test_plan_reads_exactly_the_designs_tensors():
    from grout_b200.engine.model import expected_tensors
    exp = expected_tensors(_plan(CFG))
    shapes = {n: tuple(s.shape) for n, s in exp.items()}
    assert shapes["embed"] == (50, 16) and "head" not in shapes and shapes["final.norm"] == (16,)
    assert shapes["l0.norm1"] == shapes["l0.norm2"] == (16,) and "l1.norm2" not in shapes and "l1.hc2.in" not in shapes
    assert shapes["l0.hc1.in"] == shapes["l0.hc2.out"] == (3,) and shapes["l2.hc2.mix"] == (3, 3)
    assert shapes["l0.mix.q"] == (24, 16) and shapes["l0.mix.k"] == (12, 16) and "l0.mix.v" not in shapes
    assert shapes["l0.mix.q.b"] == (24,) and shapes["l0.mix.k.conv"] == (12, 3) and shapes["l0.mix.o"] == (16, 24)
    assert shapes["l1.mix.dq"] == (10, 16) and shapes["l1.mix.dq.norm"] == (10,) and shapes["l1.mix.uq"] == (24, 10)
    assert shapes["l1.mix.dkv"] == (12, 16) and shapes["l1.mix.uk"] == (24, 12) and shapes["l1.mix.uv"] == (12, 12)
    assert shapes["l1.mix.sink"] == (3,) and shapes["l1.mix.g"] == (12, 16) and "l1.mix.q" not in shapes
    assert shapes["l2.mix.q"] == shapes["l2.mix.k"] == (16, 16) and shapes["l2.mix.v.conv"] == (24, 4)
    assert shapes["l2.mix.A_log"] == (4,) and shapes["l2.mix.dt_bias"] == (32,) and shapes["l2.mix.norm"] == (6,)
    assert shapes["l2.mix.a2"][0] == 32 and shapes["l2.mix.g2"][0] == 24 and exp["l2.mix.a1"].free == (0,)
    assert len(shapes) == 2 + (2 + 6 + 7 + 3) + (1 + 3 + 10) + (2 + 6 + 15 + 3)


def test_inner_sizes_are_those_of_the_tensors():
    """Thin products may have any inner size; both halves must agree; nothing else is free."""
    from grout_b200.engine.model import Model, expected_tensors
    from grout_b200.parts import BuildContext
    from grout_b200.weights import random_tensors
    from grout_b200.weights.loader import WeightError, check_names_and_shapes, place
    exp = expected_tensors(_plan(CFG))
    w = dict(random_tensors(exp, 3))
    for n, axis, size in (("a1", 0, 5), ("a2", 1, 5), ("g1", 0, 11), ("g2", 1, 11)):
        shape = list(w["l2.mix." + n].shape)
        shape[axis] = size
        w["l2.mix." + n] = torch.randn(shape).bfloat16()
    shapes = lambda: {n: tuple(t.shape) for n, t in w.items()}
    check_names_and_shapes(exp, shapes())
    model = Model(_plan(CFG), BuildContext(torch.bfloat16, torch.device("cpu")))
    get = lambda n: place(w[n], exp[n], torch.bfloat16, "cpu")
    model.load(get)
    mixer = model.blocks[2].mixer
    assert mixer.n_low == 16 and mixer.thin.weight.shape == (32 + 24, 16)      # filled up to whole eights
    x = torch.randn(3, 16).bfloat16().double()
    low = x @ mixer.proj.weight[-16:].double().T
    wide = low @ mixer.thin.weight.double().T
    d = {n: w["l2.mix." + n].double() for n in ("a1", "a2", "g1", "g2")}
    assert torch.allclose(wide[:, :32], (x @ d["a1"].T) @ d["a2"].T) and torch.allclose(wide[:, 32:], (x @ d["g1"].T) @ d["g2"].T)
    w["l2.mix.a2"] = torch.zeros(32, 6).bfloat16()
    with pytest.raises(ValueError, match="inner sizes"):
        model.load(get)
    w["l2.mix.a2"] = torch.zeros(31, 5).bfloat16()
    with pytest.raises(WeightError, match="l2.mix.a2"):
        check_names_and_shapes(exp, shapes())


def test_needs_of_the_cache():
    from grout_b200.cache import KVSpec, SequenceCache, SideBySideSpec, StateSpec
    from grout_b200.engine.model import Model
    from grout_b200.parts import BuildContext
    model = Model(_plan(CFG), BuildContext(torch.float32, torch.device("cpu")))
    specs = [b.cache_spec() for b in model.blocks]
    assert specs[0] == SideBySideSpec((KVSpec(2, 6, 5), StateSpec((2 * 36,))))     # two kept inputs of 36 channels
    assert specs[1] == KVSpec(1, 12, None, values_in_keys=True)
    assert specs[2] == StateSpec((3 * (16 + 16 + 24) + 4 * 8 * 6,))
    half = Model(_plan(CFG), BuildContext(torch.bfloat16, torch.device("cpu")))
    assert [half.blocks[0].cache_spec().specs[0].head_dim, half.blocks[1].cache_spec().head_dim] == [16, 16]
    one = dict(CFG, layers=[dict(type="attention", mixer=dict(ATT, conv=1), mlp=None)])
    assert Model(_plan(one), BuildContext(torch.float32, torch.device("cpu"))).blocks[0].cache_spec() == KVSpec(2, 6, 5)
    cache = SequenceCache(model.cache_layout(), max_tokens=640, max_slots=3, max_seq_len=512, dtype=torch.float32, device="cpu")
    a = cache.open()
    cache.reserve(a, 200)
    cache.advance(a, 200)
    window = cache.stores[0].stores
    assert window[0].pool.n_held == 1 and cache.stores[1].pool.n_held == 4         # position 200 sees 196..
    window[1].state[0, a] = 5.0
    cache.stores[2].state[0, a] = 7.0
    cache.close(a)
    assert cache.open() == a                                  # the slot is used again: its states start from zeros
    assert not window[1].state[0, a].any() and not cache.stores[2].state[0, a].any()
    cache.check()


def test_random_weights_of_mixing_matrices_lie_near_the_identity():
    from grout_b200.parts import ParamSpec
    from grout_b200.weights.random_init import random_tensor
    m = random_tensor("x", ParamSpec((40, 40), "mixing"), 1, torch.float32)
    assert abs(float(m.diagonal().mean()) - 1.0) < 0.1 and abs(float((m - torch.eye(40)).std()) - 0.1) < 0.02


def test_streams_by_hand():
    X = torch.tensor([[[1.0, 2.0]], [[3.0, 5.0]]], dtype=torch.float64)
    assert plain.read_streams(X, torch.tensor([2.0, -1.0])).tolist() == [[-1.0, -1.0]]
    M, b, y = torch.tensor([[1.0, 10.0], [100.0, 1000.0]]), torch.tensor([0.5, 2.0]), torch.tensor([[4.0, 6.0]], dtype=torch.float64)
    new = plain.write_streams(X, M, b, y)                      # stream t: sum_s M[s, t] X_s + b_t y
    assert new.tolist() == [[[1 + 300 + 2.0, 2 + 500 + 3.0]], [[10 + 3000 + 8.0, 20 + 5000 + 12.0]]]


def test_convolution_and_rotation_by_hand():
    x, w = torch.tensor([[1.0], [2.0], [4.0]]), torch.tensor([[7.0, 5.0, 3.0]])
    assert plain.short_conv(x, w).flatten().tolist() == [3.0, 6.0 + 5.0, 12.0 + 10.0 + 7.0]    # the last tap is the current row's
    v = torch.arange(1.0, 7.0).view(1, 1, 6)
    r = plain.rotate_halves(v, [3], 100.0, 4)[0, 0]
    for i, f in ((0, 1.0), (1, 0.1)):
        c, s = math.cos(3 * f), math.sin(3 * f)
        assert math.isclose(r[i], (i + 1) * c - (i + 3) * s) and math.isclose(r[i + 2], (i + 3) * c + (i + 1) * s)
    assert r[4:].tolist() == [5.0, 6.0]


def test_attention_by_hand():
    q = torch.tensor([[1.0], [1.0], [1.0]])
    k, v = torch.tensor([[2.0], [1.0], [-1.0]]), torch.tensor([[10.0], [20.0], [40.0]])
    mask = plain.sees_window(3, 2)
    assert mask.tolist() == [[True, False, False], [True, True, False], [False, True, True]]
    e = lambda s: math.exp(1.5 * math.tanh(0.5 * s / 1.5))
    out = plain.softmax_attention(q, k, v, 0.5, mask, cap=1.5)
    assert math.isclose(out[2], (e(1) * 20 + e(-1) * 40) / (e(1) + e(-1)))
    out = plain.softmax_attention(q, k, v, 0.5, plain.sees_window(3, None), sink=0.7)
    den = math.exp(1.0) + math.exp(0.5) + math.exp(-0.5) + math.exp(0.7)
    assert math.isclose(out[2], (math.exp(1.0) * 10 + math.exp(0.5) * 20 + math.exp(-0.5) * 40) / den)


def test_delta_rule_by_hand():
    g = torch.tensor([[0.5, 0.25]], dtype=torch.float64)
    S0 = torch.tensor([[2.0], [4.0]], dtype=torch.float64)
    k, q, v = (torch.tensor([x], dtype=torch.float64) for x in ([0.6, 0.8], [1.0, 2.0], [3.0]))
    o, S = plain.delta_head(q, k, v, torch.tensor([0.5], dtype=torch.float64), g, S0)
    u = 0.5 * (3.0 - (0.6 * 1.0 + 0.8 * 1.0))                  # the state has faded to (1, 1) before it is read
    assert math.isclose(S[0], 1.0 + 0.6 * u) and math.isclose(S[1], 1.0 + 0.8 * u)
    assert math.isclose(o[0], S[0] + 2 * S[1])                 # the read-out sees the row's own write
    w = {"a1": torch.tensor([[1.0]]), "a2": torch.tensor([[1.0], [2.0], [3.0], [4.0]]), "dt_bias": torch.tensor([0.1, 0.2, 0.3, 0.4]),
         "A_log": torch.tensor([0.0, 1.0])}
    d = plain.channel_decays(torch.tensor([[0.5]]), w, "", 2, 2)[0]
    for h in range(2):
        for c in range(2):
            i = 2 * h + c
            z = math.log1p(math.exp(0.5 * (i + 1) + 0.1 * (i + 1)))
            assert math.isclose(d[h, c], math.exp(-math.exp(float(h)) * z), rel_tol=1e-6)


def test_layers_without_feed_forward_and_the_sum_at_the_end():
    from grout_b200.engine.model import expected_tensors
    from grout_b200.weights import random_tensors
    w = dict(random_tensors(expected_tensors(_plan(CFG)), 5, torch.float32))
    toks = [3, 7, 7, 49, 0, 12]
    out, after = plain.forward(toks, w, CFG, return_layers=True)
    assert out.shape == (6, 50) and after.shape == (3, 6, 16)
    last = plain.rms_norm(after[-1], w["final.norm"], 1e-5) @ w["embed"].double().T    # the table without its scale
    assert torch.allclose(out, last)
    again = plain.forward(toks[:4], w, CFG)
    assert torch.allclose(out[:4], again)
