"""The Keralix design through the engine against the plain implementation, in every way of
cutting the work, on four small models that differ in every size and constant (and from
layer to layer): one to five residual streams, the mixers in different orders with and
without feed-forwards, windows from two tokens to longer than any request and none, rotations
of a whole head, of a part and none, with and without capped scores, one tap to more taps
than a portion has rows, several heads on one key, values narrower and wider than keys,
latents of every size, sizes that take the tcgen05 and TMA attention kernels, the mma.sync ones
and the plain one, heads of the delta rule that go chunk by chunk and others that do not,
widths that are no multiple of eight.  The random weights are reshaped so that faults show:
sharp attention, sinks that weigh as much as the keys, streams that differ, states that keep
and that fade."""
import json
import os

import pytest
import torch

from conftest import random_tokens
from helpers import run_batch, run_chunks, run_schedule, run_tail_decoded, run_whole
from plain import keralix as plain

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
ROW_BAR = 0.08


def assert_close(got, want, dtype, what=""):
    """32-bit: every value within 2e-4 of the logits' spread.  bfloat16: rounding moves sharp
    attention weights in single rows while the rows as a whole stay close; the bar is on the
    median and the upper quartile of the rows' differences (root mean square, mean taken off)
    as a share of that spread.  A lost mechanism, a wrong page or a lost state moves every row
    after it by more than 0.3."""
    got, want = got.detach().double().cpu(), want.detach().double().cpu()
    assert got.shape == want.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(want.shape)}"
    spread = float((want - want.mean(dim=-1, keepdim=True)).pow(2).mean().sqrt())
    d = got - want
    if dtype == "float32":
        assert float(d.abs().max()) <= 1e-3 * spread, f"{what}: max err {float(d.abs().max()):.3g} of {spread:.3g}"
        return
    rows = (d - d.mean(dim=-1, keepdim=True)).pow(2).mean(dim=-1).sqrt() / spread
    med, q3 = float(rows.median()), float(rows.quantile(0.75))
    assert med <= ROW_BAR and q3 <= 2 * ROW_BAR, (
        f"{what}: median row differs by {med:.3f} of the logits' spread, upper quartile {q3:.3f}, "
        f"worst {float(rows.max()):.3f} (row {int(rows.argmax())})")


def _att(heads, kv_heads, dim, conv, scale, size=None, cap=None, rot=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, conv=conv, scale=scale)
    if size:
        m["mask"] = {"size": size}
    if cap:
        m["softcap"] = cap
    if rot:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    return m


def _lat(heads, dim, vdim, q_rank, kv_rank, scale):
    return dict(heads=heads, dim=dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale)


def _delta(heads, kv_heads, dim, vdim, conv):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)


def _layer(kind, mixer, ff=None):
    return dict(type={"A": "attention", "L": "latent_attention", "D": "channel_delta"}[kind], mixer=mixer,
                mlp={"kind": "dense", "ff": ff} if ff else None)


KER = {
    # a window shorter than a page, rotation of a part, three streams
    "T": dict(architecture="Keralix", vocab=211, width=64, streams=3, norm={"eps": 1e-5}, embedding={"scale": 3.0}, layers=[
        _layer("A", _att(4, 2, 32, 3, 0.4, 9, 20.0, (1e4, 16)), 96),
        _layer("D", _delta(4, 2, 16, 24, 4)),
        _layer("L", _lat(4, 16, 24, 40, 48, 0.3), 72),
        _layer("D", _delta(2, 2, 32, 16, 2), 48)]),
    # heads of 64 and latents of 64 (the tcgen05 prompt kernel, the TMA decode kernel from 64 pairs on), windows
    # longer than a page, a latent attention of more than sixteen heads
    "U": dict(architecture="Keralix", vocab=300, width=128, streams=4, norm={"eps": 3e-6}, embedding={"scale": 8.0}, layers=[
        _layer("D", _delta(3, 1, 64, 64, 3), 64),
        _layer("A", _att(8, 4, 64, 4, 0.15, 70, 50.0, (1e6, 64)), 96),
        _layer("L", _lat(20, 16, 16, 24, 64, 0.2)),
        _layer("A", _att(4, 4, 64, 2, 0.2, 130, 8.0, (500.0, 32))),
        _layer("L", _lat(2, 64, 32, 96, 128, 0.1), 160)]),
    # odd sizes, no window, no cap, no rotation, one tap, five streams
    "V": dict(architecture="Keralix", vocab=160, width=96, streams=5, norm={"eps": 1e-4}, embedding={"scale": 2.0}, layers=[
        _layer("L", _lat(3, 20, 12, 33, 150, 0.2), 40),
        _layer("A", _att(6, 2, 20, 5, 0.15, None, 5.0, (1e3, 20)), 88),
        _layer("D", _delta(3, 3, 20, 10, 1), 24),
        _layer("A", _att(3, 1, 24, 1, 0.15, 65, None, None)),
        _layer("D", _delta(2, 1, 33, 36, 9)),
        _layer("A", _att(5, 5, 17, 12, 0.13, 2, 12.0, (1e5, 6)), 16)]),
    # nothing a multiple of eight; one stream
    "W": dict(architecture="Keralix", vocab=173, width=100, streams=1, norm={"eps": 2e-5}, embedding={"scale": 10.0}, layers=[
        _layer("D", _delta(5, 5, 12, 20, 3), 52),
        _layer("L", _lat(5, 12, 28, 20, 36, 0.4)),
        _layer("A", _att(3, 3, 44, 3, 0.25, 64, 30.0, (50.0, 12)), 36)]),
}
SEEDS = {"T": 11, "U": 13, "V": 17, "W": 19}
LENGTHS = {"T": [1, 5, 70, 150], "U": [2, 64, 129, 300], "V": [3, 131, 210], "W": [1, 66, 200]}


def _sharpen(tensors):
    out = {}
    for name, t in tensors:
        f = t.float()
        if name == "embed":
            f = f * 40.0
        elif name.endswith((".mix.q", ".mix.k", ".mix.uq", ".mix.uk")):
            f = f * 12.0                                        # sharp attention: single keys carry a row
        elif name.endswith((".mix.dq", ".mix.dkv", ".mix.v", ".mix.uv", ".mix.g", ".mix.b", ".mix.a1", ".mix.a2",
                            ".mix.g1", ".mix.g2")):
            f = f * 8.0
        elif name.endswith(".mix.o"):
            f = f * 6.0
        elif name.endswith(".conv"):
            f = f - 1.0 + 6.0 * (f - 1.0)                       # taps on both sides of zero
            f[:, -1] += 1.0
        elif name.endswith(".sink"):
            f = f * 20.0 + 1.0
        elif name.endswith((".A_log", ".dt_bias")):
            f = f * 15.0 - 1.0                                  # channels that keep and channels that fade
        elif name.endswith((".q.b", ".k.b")):
            f = f * 4.0
        elif ".hc" in name:
            f = f * 0.7 if name.endswith(".mix") else f * 0.8
        elif ".mlp." in name:
            f = f * 6.0                                         # feed-forwards that weigh as much as the mixers
        out[name] = f.to(t.dtype)
    return out


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (folder, config dict, {tensor name: CPU tensor})."""
    import grout_b200.architectures  # noqa: F401
    from grout_b200.config import resolve_architecture
    from grout_b200.engine.model import expected_tensors
    from grout_b200.weights import random_tensors, write_safetensors
    base = tmp_path_factory.mktemp("keralix")
    out = {}
    for name, cfg in KER.items():
        arch = resolve_architecture(cfg)
        exp = expected_tensors(arch.plan(arch.config_cls.from_dict(cfg)))
        w = _sharpen(random_tensors(exp, SEEDS[name]))
        for n in [n for n in w if n.endswith(".a1")]:           # inner sizes that no configuration states
            w[n], w[n[:-1] + "2"] = w[n][:-3].clone(), w[n[:-1] + "2"][:, :-3].clone()
        folder = str(base / name)
        os.makedirs(folder)
        with open(os.path.join(folder, "config.json"), "w") as fh:
            json.dump(cfg, fh)
        write_safetensors(os.path.join(folder, "model.safetensors"), list(w.items()))
        out[name] = (folder, cfg, w)
    return out


@pytest.fixture(scope="module")
def engines(models):
    from grout_b200.engine import Engine
    made = {}

    def get(name, dtype, **kw):
        key = (name, dtype, tuple(sorted(kw.items())))
        if key not in made:
            made[key] = Engine.load(models[name][0], dtype=dtype, max_tokens=4096, max_batch=8,
                                    max_seq_len=512, **kw)
        return made[key]
    return get


@pytest.fixture(scope="module")
def oracle(models):
    memo = {}

    def get(name, tokens):
        key = (name, tuple(tokens))
        if key not in memo:
            _d, cfg, w = models[name]
            memo[key] = plain.logits(w, cfg, list(tokens))
        return memo[key]
    return get


def test_the_sharpened_weights_do_what_they_are_for(models):
    """Models on which a window one token off, a lost cap, rotation, sink, bias, tap, gate, stream or
    fading state shows in the logits."""
    def moved(name, t, fn=None, change=None):
        """The largest change of a logit, as a share of the logits' spread."""
        _d, c0, w0 = models[name]
        c, w = json.loads(json.dumps(c0)), w0
        if fn:
            fn(c["layers"])
        if change:
            end, f = change
            w = {k: (f(v.float()) if k.endswith(end) else v) for k, v in w0.items()}
        ref = plain.logits(w0, c0, t)
        return float((plain.logits(w, c, t) - ref).abs().max() / ref.std())

    tt, tu = random_tokens(60, KER["T"]["vocab"], 1), random_tokens(150, KER["U"]["vocab"], 2)
    for d in (-1, 1):
        assert moved("T", tt, lambda L: L[0]["mixer"]["mask"].update(size=9 + d)) > 0.1
        assert moved("U", tu, lambda L: L[1]["mixer"]["mask"].update(size=70 + d)) > 0.1
        assert moved("U", tu, lambda L: L[3]["mixer"]["mask"].update(size=130 + d)) > 0.1
    assert moved("T", tt, lambda L: L[0]["mixer"].pop("softcap")) > 0.1
    assert moved("T", tt, lambda L: L[0]["mixer"].pop("rot")) > 0.1
    for end, f in ((".sink", lambda v: v - 40), (".q.b", torch.zeros_like), (".k.b", torch.zeros_like),
                   (".dt_bias", lambda v: v + 0.2), (".A_log", lambda v: v + 0.2), (".g2", torch.zeros_like),
                   (".mix.b", torch.zeros_like), (".dq.norm", torch.ones_like), (".dkv.norm", torch.ones_like),
                   (".mix.norm", torch.ones_like), ("hc1.mix", lambda v: v.T.contiguous()), ("hc2.mix", torch.eye(3).mul),
                   ("hc1.out", torch.ones_like), ("hc2.in", torch.ones_like)):
        assert moved("T", tt, change=(end, f)) > 0.05, end
    first_tap = lambda v: torch.cat([torch.zeros_like(v[:, :1]), v[:, 1:]], 1)
    for end in (".q.conv", ".k.conv", ".v.conv"):
        assert moved("T", tt, change=(end, first_tap)) > 0.1, end


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(KER))
def test_each_request_alone_and_whole(engines, oracle, name, dtype):
    eng = engines(name, dtype)
    for i, n in enumerate(LENGTHS[name]):
        toks = random_tokens(n, KER[name]["vocab"], 100 + i)
        assert_close(run_whole(eng, toks), oracle(name, toks), dtype, f"{name} whole, {n} tokens")
    eng.cache.check()
    assert eng.cache.slots.n_held == 0 and eng.cache.tokens_held() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(KER))
def test_prefill_against_token_by_token(engines, oracle, name, dtype):
    """The tail decoded across a window's and a page's edge; then everything but the first token
    decoded, so that every edge is passed in single steps too."""
    eng = engines(name, dtype)
    toks = random_tokens(LENGTHS[name][-1], KER[name]["vocab"], 200)
    assert_close(run_tail_decoded(eng, toks, tail=40), oracle(name, toks), dtype, f"{name} tail")
    short = toks[:90]
    assert_close(run_tail_decoded(eng, short, tail=89), oracle(name, short), dtype, f"{name} decoded from the first token")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(KER))
def test_a_prompt_fed_in_portions(engines, oracle, name, dtype):
    """Portions of two tokens and of one (shorter than the convolutions and the windows); portions that
    end one short of a page and of a chunk of the delta rule, on it and beyond it."""
    eng = engines(name, dtype)
    for i, chunks in enumerate([[2] * 12 + [1, 3], [63, 1, 64, 2], [60, 10, 70, 61], [1, 1, 1, 2, 1, 30, 1, 1],
                                [31, 33, 96, 1, 32]]):
        toks = random_tokens(sum(chunks), KER[name]["vocab"], 700 + i)
        assert_close(run_chunks(eng, toks, chunks), oracle(name, toks), dtype, f"{name} portions {chunks}")
    eng.cache.check()
    assert eng.cache.slots.n_held == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(KER))
def test_unequal_batches_one_after_another(engines, oracle, name, dtype):
    """Three batches in a row on one engine: slots (and with them the states' rows and the kept inputs of
    the convolutions) and pages of an earlier batch are used again by a later one, and within a batch
    the shorter requests end earlier.  Each request as in a run of its own."""
    eng = engines(name, dtype)
    V = KER[name]["vocab"]
    plans = [[(5, 3), (11, 9), (17, 1)],
             [(1, 20), (7, 2), (30, 11), (64, 5), (130, 33), (200, 30)],
             [(65, 4), (2, 4), (128, 70)]]
    for b, plan in enumerate(plans):
        reqs = [random_tokens(p + d, V, 300 + 10 * b + i) for i, (p, d) in enumerate(plan)]
        got = run_batch(eng, reqs, [p for p, _ in plan])
        for i, r in enumerate(reqs):
            assert_close(got[i], oracle(name, r), dtype, f"{name} batch {b} request {i}")
            if dtype == "float32":
                assert_close(got[i], run_whole(eng, r), dtype, f"{name} batch {b} request {i} against itself alone")
        eng.cache.check()
        assert eng.cache.slots.n_held == 0 and eng.cache.tokens_held() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["T", "U"])
def test_first_tokens_and_long_decoding(engines, oracle, name, dtype):
    """A prompt of one token and 330 decoded ones: the first positions (convolutions and windows that are
    not full yet, an empty state) and a long run of single steps across page and window borders,
    with stores that give pages back."""
    eng = engines(name, dtype)
    toks = random_tokens(331, KER[name]["vocab"], 400)
    assert_close(run_tail_decoded(eng, toks, tail=330), oracle(name, toks), dtype, "long decoding")
    eng.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(KER))
def test_steps_that_mix_one_and_many_tokens(engines, oracle, name, dtype):
    eng = engines(name, dtype)
    lengths = [20 + 5 + 1 + 3 + 1, 9 + 1 + 1 + 1 + 1 + 1, 70 + 1 + 2]
    schedule = [{0: 20, 1: 9}, {0: 5, 1: 1}, {0: 1, 1: 1, 2: 70}, {0: 3, 1: 1, 2: 1}, {0: 1, 1: 1, 2: 2}, {1: 1}]
    reqs = [random_tokens(n, KER[name]["vocab"], 720 + i) for i, n in enumerate(lengths)]
    got = run_schedule(eng, reqs, schedule)
    for i, r in enumerate(reqs):
        assert_close(got[i], oracle(name, r), dtype, f"{name} mixed steps, request {i}")
    eng.cache.check()
    assert eng.cache.slots.n_held == 0


def test_windowed_stores_give_pages_back(engines):
    eng = engines("U", "float32")
    s = eng.open_sequence()
    eng.step([(s, random_tokens(500, KER["U"]["vocab"], 410))], [[0]])
    pools = [st.pool for g in eng.cache.stores for st in getattr(g, "stores", [g]) if hasattr(st, "pool")]
    # the latent attentions keep all eight pages; position 500 looks back 70 (pages 6, 7) and 130 (5 to 7)
    assert sorted(p.n_held for p in pools) == [2, 3, 8, 8]
    eng.close_sequence(s)
    eng.cache.check()
    assert eng.cache.tokens_held() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_captured_steps_against_steps_launched_one_by_one(engines, oracle, dtype):
    reqs = [random_tokens(n, KER["U"]["vocab"], 740 + i) for i, n in enumerate((90, 33, 140))]
    outs = {}
    for use in (True, False):
        eng = engines("U", dtype, use_graphs=use)
        outs[use] = run_batch(eng, reqs, [60, 30, 100])
    for i, r in enumerate(reqs):
        for use in (True, False):
            assert_close(outs[use][i], oracle("U", r), dtype, f"graphs {use}, request {i}")


def test_many_sequences_take_the_tma_decode_kernel(models, oracle):
    """Sixteen sequences of four kv heads are 64 (sequence, kv head) pairs: decode steps of heads of 64
    then run on the TMA kernel."""
    from grout_b200.engine import Engine
    folder, cfg, _w = models["U"]
    eng = Engine.load(folder, dtype="bfloat16", max_tokens=16 * 512, max_batch=16, max_seq_len=512)
    reqs = [random_tokens(150 + 7 * i, cfg["vocab"], 760 + i) for i in range(16)]
    got = run_batch(eng, reqs, [len(r) - 12 for r in reqs])
    for i in (0, 5, 15):
        assert_close(got[i], oracle("U", reqs[i]), "bfloat16", f"request {i} of 16")
    eng.cache.check()


@pytest.mark.parametrize("name", sorted(KER))
def test_greedy_generation_through_the_engine(models, name):
    """Engine.generate (its scheduler, cache and device sampler) against the plain loop, in 32-bit,
    where the argmax is the same token."""
    from grout_b200.engine import Engine
    folder, cfg, w = models[name]
    eng = Engine.load(folder, dtype="float32", max_tokens=2048, max_batch=3)
    prompts = [random_tokens(n, cfg["vocab"], 800 + i) for i, n in enumerate((1, 7, 30, 64, 5))]
    want = [plain.greedy_generate(w, cfg, p, 8) for p in prompts]
    outs = eng.generate(prompts, 8, ignore_eos=True)            # five requests on three slots
    assert [o.token_ids for o in outs] == want
    stop = want[1][3]
    outs = eng.generate(prompts, 8, stop_ids=[stop])
    assert [o.token_ids for o in outs] == [w_[:w_.index(stop)] if stop in w_ else w_ for w_ in want]
    eng.cache.check()
    assert eng.cache.slots.n_held == 0 and eng.cache.tokens_held() == 0


def test_generation_in_bfloat16_and_the_command_line(models, tmp_path):
    """bfloat16 generation runs through captured steps; its tokens are the plain loop's wherever the
    plain logits leave no doubt.  And the command line serves the design as it serves the others."""
    import subprocess
    import sys
    from conftest import ROOT
    from grout_b200.engine import Engine
    folder, cfg, w = models["U"]
    eng = Engine.load(folder, dtype="bfloat16", max_tokens=2048, max_batch=4)
    prompt = random_tokens(70, cfg["vocab"], 820)
    got = eng.generate([prompt], 10, ignore_eos=True)[0].token_ids
    seq = list(prompt)
    for tok in got:
        row = plain.logits(w, cfg, seq, rows=[len(seq) - 1])[0]
        top2 = torch.topk(row, 2).values
        if float(top2[0] - top2[1]) > 0.3 * float(row.std()):
            assert tok == int(torch.argmax(row)), len(seq)
        seq.append(tok)
    out = tmp_path / "out.json"
    ids = ",".join(str(t) for t in prompt[:9])
    r = subprocess.run([sys.executable, "-m", "grout_b200", "--model", folder, "--prompt-ids", ids,
                        "--max-new-tokens", "6", "--ignore-eos", "--fp32", "--device-argmax",
                        "--output-json", str(out), "--quiet"], cwd=ROOT, capture_output=True, text=True)
    assert r.returncode == 0, r.stderr[-2000:]
    assert json.load(open(out))["token_ids"] == plain.greedy_generate(w, cfg, prompt[:9], 6)


def test_trace_replay_serves_the_design(models, tmp_path):
    """bin/trace_run on a Keralix folder: a prompt, then single tokens, two requests."""
    import subprocess
    import sys
    import numpy as np
    from conftest import ROOT
    folder, cfg, w = models["T"]
    a, b = random_tokens(40, cfg["vocab"], 840), random_tokens(9, cfg["vocab"], 841)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:37], "want": [0, 36]},
                                     {"id": "b", "tokens": b[:8], "want": [7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [a[37]], "want": []},
                                     {"id": "b", "tokens": [b[8]], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": [a[38]], "want": [0]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": [a[39]], "want": [0]}], "end": ["a"]}]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder,
                        "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "128"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    la, lb = plain.logits(w, cfg, a), plain.logits(w, cfg, b)
    want = {0: torch.stack([la[0], la[36], lb[7]]), 1: lb[8:9], 2: la[38:39], 3: la[39:40]}
    for i, wnt in want.items():
        got = torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"]))
        assert_close(got, wnt, "float32", f"step {i}")
