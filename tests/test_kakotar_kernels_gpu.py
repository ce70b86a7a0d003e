"""Each mechanism that the Kakotar design brought, alone, against the plain implementation's
function for it: the dynamic tanh with the sum in front of it, YaRN-stretched rotations, two
maps a cached row in the q/k kernel, attention in chunks (planted keys on both sides of a
chunk's and a page's border, in prompts and in single steps, through every attention kernel),
the difference of two maps, lightning attention (state carried over steps, slots used again,
padding rows, long prompts chunk by chunk), layers that read another layer's keys, and
ungated experts with corrected sigmoid scores, groups by their two largest, normalised
weights and a shared expert."""
import math

import pytest
import torch

from plain import kakotar as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
TOL = {torch.float32: dict(atol=3e-5, rtol=3e-4), torch.bfloat16: dict(atol=0.03, rtol=0.03)}
DTYPES = [torch.float32, torch.bfloat16]


def close(got, want, dtype, what="", scale=1.0):
    """``scale``: the size of the terms whose sum the value is (their rounding is what is left
    where they cancel)."""
    got, want = got.detach().double().cpu(), want.detach().double().cpu()
    assert got.shape == want.shape, (what, got.shape, want.shape)
    err = (got - want).abs()
    bound = TOL[dtype]["atol"] * max(1.0, float(scale)) + TOL[dtype]["rtol"] * want.abs()
    assert bool((err <= bound).all()), f"{what}: max err {err.max().item():.3g} at {int(err.argmax())}"


def rows_close(got, want, what="", most=0.03):
    """bfloat16 results of several roundings: the difference's root mean square, and its largest."""
    d = got.detach().double().cpu() - want.double()
    assert float(d.pow(2).mean().sqrt() / want.pow(2).mean().sqrt()) < most, what
    assert float(d.abs().max()) < 6 * most * float(want.abs().max()), what


def rnd(*shape, seed=0, scale=1.0, dtype=torch.float32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def make_step(seqs):
    """The fields of a step that the kernels read, for sequences given as (slot, start, n)."""
    from grout_b200.engine.batch import make_context
    return make_context([(s, st, [0] * n) for s, st, n in seqs], None, DEV)


def make_part(family, kind, dtype, **args):
    from grout_b200.parts import BuildContext, PartSpec, build_part
    return build_part(family, PartSpec(kind, args), BuildContext(dtype, torch.device(DEV)))


g32 = lambda t: t.float().to(DEV).contiguous()


# ------------------------------------------------------------------ dynamic tanh
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,N,parts", [(1, 96, 0), (5, 100, 3), (3, 7, 2), (70, 2560, 1), (514, 640, 13), (2, 4099, 9)])
def test_dynamic_tanh_with_the_sum_in_front(dtype, T, N, parts):
    w = {"n": 1 + rnd(N, seed=1, scale=0.3), "n.b": rnd(N, seed=2, scale=0.5), "n.alpha": torch.tensor(0.7)}
    w = {k: v.to(dtype) for k, v in w.items()}
    norm = make_part("norm", "dynamic_tanh", dtype, dim=N, name="n")
    norm.load({k: v.to(DEV) for k, v in w.items()})
    res = rnd(T, N, seed=3, scale=3.0)
    delta = rnd(T, N, seed=4).to(dtype)
    x = res.double() + delta.double()
    got_res, y = norm.add_norm(res.to(DEV), delta.to(DEV))
    assert got_res.dtype == torch.float32 and y.dtype == dtype
    close(got_res, x, torch.float32, "sum")
    close(y, plain.dynamic_tanh(x, w, "n"), dtype, "norm")
    if parts:                       # a stack of 32-bit partial sums, and a gather of rows in another order
        stack = rnd(parts, T, N, seed=5)
        x = res.double() + stack.double().sum(0)
        rows = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32)
        before = res.to(DEV)
        got_res, y = norm.add_norm(before, stack.to(DEV), rows=rows.to(DEV))
        close(got_res, x[rows.long()], torch.float32, "rows of the sum")
        close(y, plain.dynamic_tanh(x[rows.long()], w, "n"), dtype, "rows")
        assert torch.equal(before.cpu(), res)          # with a row list the stream stays as it is
        _r, y = norm.add_norm(None, stack.to(DEV))     # a stream that starts with the contribution
        close(y, plain.dynamic_tanh(stack.double().sum(0), w, "n"), dtype, "no stream before")
    close(norm.forward(delta.to(DEV)), plain.dynamic_tanh(delta, w, "n"), dtype, "alone")


def test_dynamic_tanh_saturates_and_takes_every_kind_of_contribution():
    from grout_b200.parts import Contribution
    N, T = 24, 6
    w = {"n": torch.ones(N), "n.b": torch.zeros(N), "n.alpha": torch.tensor(-4.0)}
    norm = make_part("norm", "dynamic_tanh", torch.float32, dim=N, name="n")
    norm.load({k: v.to(DEV) for k, v in w.items()})
    x = rnd(T, N, seed=1, scale=1e4)
    _r, y = norm.add_norm(x.to(DEV), None)             # large arguments: exactly -1 and 1
    assert torch.equal(y.cpu().sign(), -x.sign()) and float((y.abs() - 1).abs().max()) == 0.0
    a, b = rnd(T, N, seed=2), rnd(2, T, N, seed=3)
    x = rnd(T, N, seed=4, scale=0.3)
    want = x.double() + 0.5 * a.double() + b.double().sum(0)
    res, y = norm.add_norm(x.to(DEV), (Contribution(a.to(DEV), mult=0.5), b.to(DEV)))
    close(res, want, torch.float32)
    close(y, plain.dynamic_tanh(want, w, "n"), torch.float32)


# ------------------------------------------------------------------ rotation
SCALINGS = [dict(factor=4.0, original=64, fast=8.0, slow=1.0), dict(factor=1.0, original=1024, fast=32.0, slow=1.0),
            dict(factor=7.5, original=4, fast=32.0, slow=30.0),          # the ramp shrinks to nothing
            dict(factor=16.0, original=10 ** 9, fast=2.0, slow=1.0),     # ... and lies beyond the last element
            dict(factor=3.0, original=96, low=1.0, high=4.0), None]


@pytest.mark.parametrize("scaling", SCALINGS)
def test_rotation_tables_and_the_qk_kernel(scaling):
    from grout_b200.kernels import ops
    for D, dims, base, H, G in ((64, 64, 5e5, 3, 1), (32, 12, 300.0, 2, 2), (96, 96, 1e4, 2, 1), (128, 128, 1e6, 4, 2)):
        part = make_part("position", "rotary_half_split", torch.float32, head_dim=D, theta=base, rot_dim=dims,
                         scaling=scaling, exact_table=True)
        rot = part.rotary()
        f, amp = plain.rotation_of(dict(base=base, dims=dims, scaling=scaling))
        assert abs(rot.amplitude - amp) < 1e-12
        assert torch.allclose(rot.inv_freq.double().cpu(), torch.tensor(f, dtype=torch.float64), rtol=1e-7, atol=0)
        for dtype in DTYPES:
            for T, start in ((3, 0), (140, 37)):
                qkv = rnd(T, (H + 2 * G) * D, seed=T).to(dtype)
                step = make_step([(-1, start, T)])
                q, kv = ops.qk_prepare(qkv.to(DEV), H, G, D, inv_freq=rot.inv_freq, rot_dim=dims,
                                       rot_scale=rot.amplitude, token_seq=step.token_seq, token_pos=step.token_pos,
                                       slots=step.slots, want_kv_out=True)
                src, pos = qkv.double().view(T, H + 2 * G, D), list(range(start, start + T))
                for got, want, nm in ((q, src[:, :H], "q"), (kv[:, :G], src[:, H:H + G], "k")):
                    close(got.float(), plain.rotate(want, pos, f, amp), dtype, f"{nm} {D} {dims}", scale=3)
                assert torch.equal(kv[:, G:].cpu(), qkv.view(T, -1, D)[:, H + G:])          # v passes


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [(4, 2, 32, 64, 32), (2, 1, 16, 48, 8), (3, 3, 24, 20, 4), (2, 2, 20, 12, 20),
                                   (8, 2, 64, 128, 64), (2, 1, 8, 8, 0)])
def test_two_maps_a_cached_row(dtype, shape):
    """The q/k kernel lays a kv head's two keys side by side into one page row and makes a query row
    per map that is zero where the other map's key lies; from the projection and from partial sums of
    it; padding rows store nothing."""
    from grout_b200.kernels import ops
    H, G, D, Dv, dims = shape
    Ds = max(2 * D, Dv)
    Ds = (Ds + 15) // 16 * 16 if dtype == torch.bfloat16 else Ds
    f, amp = plain.rotation_of(dict(base=1000.0, dims=dims, scaling=SCALINGS[0])) if dims else ([], 1.0)
    inv = torch.tensor(f, dtype=torch.float32, device=DEV) if dims else None
    page, T = 64, 90
    for n in (T, 7):
        width = 2 * H * D + 2 * G * D + G * Dv
        qkv = rnd(n, width, seed=n).to(dtype)
        stack = rnd(3, n, width, seed=n + 1)
        for given, src in ((qkv, qkv), (stack, stack.double().sum(0))) if dtype == torch.bfloat16 else ((qkv, qkv),):
            step = make_step([(1, 50, n - 3), (-1, 0, 3)])
            kp = torch.full((6, G, page, Ds), 9.0, dtype=dtype, device=DEV)
            vp = torch.full_like(kp, 9.0)
            table = torch.tensor([[0, 0, 0], [4, 2, 5]], dtype=torch.int32, device=DEV)
            q, _ = ops.qk_prepare(given.to(DEV), 2 * H, G, D, maps=2, v_dim=Dv, inv_freq=inv, rot_dim=dims,
                                  rot_scale=amp, token_seq=step.token_seq, token_pos=step.token_pos,
                                  slots=step.slots, block_table=table, k_pages=kp, v_pages=vp, page=page)
            pos = list(range(50, 50 + n - 3)) + [0, 1, 2]
            s = src.double()
            wq = plain.rotate(s[:, :2 * H * D].view(n, H, 2, D), pos, f, amp)
            wk = plain.rotate(s[:, 2 * H * D:2 * (H + G) * D].view(n, G, 2, D), pos, f, amp)
            wv = s[:, 2 * (H + G) * D:].view(n, G, Dv)
            full = torch.zeros(n, H, 2, Ds, dtype=torch.float64)
            full[:, :, 0, :D], full[:, :, 1, D:2 * D] = wq[:, :, 0], wq[:, :, 1]
            close(q, full.view(n, 2 * H, Ds), dtype, "queries", scale=3)
            stored = 0
            for t in range(n - 3):
                pg, at = int(table[1, pos[t] // page]), pos[t] % page
                kr, vr = torch.zeros(G, Ds, dtype=torch.float64), torch.zeros(G, Ds, dtype=torch.float64)
                kr[:, :2 * D], vr[:, :Dv] = wk[t].reshape(G, 2 * D), wv[t]
                close(kp[pg, :, at], kr, dtype, "keys", scale=3)
                close(vp[pg, :, at], vr, dtype, "values", scale=3)
                stored += 1
            untouched = (kp == 9.0).all(dim=-1).all(dim=1).sum()
            assert int(untouched) == 6 * page - stored


# ------------------------------------------------------------------ attention in chunks
def paged(k, v, slots_of, n_seqs, dtype, page=64, seed=7):
    """Every sequence holds keys k [T, G, D] and values v in pages in no particular order."""
    T, G, D = k.shape
    n = (T + page - 1) // page
    kp = torch.zeros(n_seqs * n + 1, G, page, D, dtype=dtype)
    vp = torch.zeros_like(kp)
    table = (torch.randperm(n_seqs * n, generator=torch.Generator().manual_seed(seed)) + 1).view(n_seqs, n).to(torch.int32)
    for sq in range(n_seqs):
        for pg in range(n):
            rows = slice(pg * page, min(T, (pg + 1) * page))
            kp[table[sq, pg], :, :rows.stop - rows.start] = k[rows].transpose(0, 1).to(dtype)
            vp[table[sq, pg], :, :rows.stop - rows.start] = v[rows].transpose(0, 1).to(dtype)
    return kp.to(DEV), vp.to(DEV), table.to(DEV)


def attention_kernels(dtype, D):
    from grout_b200.kernels import ops
    prompt, single = ["attn_generic"], ["attn_generic"]
    if dtype == torch.bfloat16 and ops.fast_attention_takes(D, 2, 2, 64):
        prompt.append("attn_prefill_bf16")
        single.append("attn_decode_bf16")
        if ops.attn_prefill_tc_takes(D, 2, 2, 64):
            prompt += ["attn_prefill_tc 128", "attn_prefill_tc 256"]
        if ops.attn_decode_tma_takes(D, 2, 2, 64):
            single.append("attn_decode_tma")
    return prompt, single


def run_attention(name, q, kp, vp, table, step, scale, **kw):
    from grout_b200.kernels import ops
    common = dict(slots=step.slots, page=64, scale=scale, **kw)
    if name == "attn_generic":
        return ops.attn_generic(q, kp, vp, table, token_seq=step.token_seq, token_pos=step.token_pos, **common)
    if name.startswith("attn_prefill_tc"):
        return ops.attn_prefill_tc(q, kp, vp, table, cu_q=step.cu_q, kv_len=step.kv_len, q_lens=step.q_lens,
                                   rows_per_block=int(name.split()[1]), **common)
    if name == "attn_prefill_bf16":
        return ops.attn_prefill_bf16(q, kp, vp, table, cu_q=step.cu_q, kv_len=step.kv_len, q_lens=step.q_lens, **common)
    fn = ops.attn_decode_bf16 if name == "attn_decode_bf16" else ops.attn_decode_tma
    return fn(q, kp, vp, table, kv_len=step.kv_len, max_kv_len=step.max_kv_len, **common)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D", [64, 128, 96, 40])
def test_a_planted_key_on_both_sides_of_a_chunk(dtype, D):
    """One query and one key that matches it among hundreds that do not, at the chunk's first position,
    the one in front of it, page borders and the query's own: it carries the row or is not seen at all.
    As a prompt's row and as a single step, with few and with many splits, through every kernel."""
    H = G = 2
    T = 330
    for chunk, at_q in ((70, 329), (64, 329), (100, 299), (100, 300), (330, 329), (500, 200), (1, 150), (7, 131), (200, 199)):
        first = at_q // chunk * chunk
        for at in sorted({first, first - 1, at_q, at_q - 1, 0, 64, 63, 128, (first + at_q) // 2}):
            if not 0 <= at <= at_q:
                continue
            k, q = rnd(T, G, D, seed=3, scale=0.05), rnd(1, H, D, seed=4, scale=0.05)
            k[at] += 3.0 * q[0] / q[0].norm(dim=-1, keepdim=True)        # a score that stands out ...
            q = q * 40.0
            v = rnd(T, G, D, seed=5)
            mask = plain.chunk_mask(T, chunk)[at_q]
            s = torch.einsum("hd,thd->ht", q[0].double(), k.double()).masked_fill(~mask[None, :], -math.inf)
            p = torch.softmax(s, dim=-1)
            want = torch.einsum("ht,thd->hd", p, v.double())
            alone = at == first and at_q == first                        # (nothing else is in sight)
            assert (float(p[0, at]) > 0.5) == (first <= at) or alone     # ... and decides the row, if it is seen
            n_seqs = 40 if dtype == torch.bfloat16 else 2
            kp, vp, table = paged(k, v, None, n_seqs, dtype)
            prompt, single = attention_kernels(dtype, D)
            bar = 0.02 if dtype == torch.float32 else 0.06
            # the query as the last of a prompt's 50 rows (rows of zeros before it)
            n = min(50, at_q + 1)
            rows = torch.zeros(n, H, D)
            rows[-1] = q[0]
            step = make_step([(1, at_q + 1 - n, n)])
            for name in prompt:
                got = run_attention(name, rows.to(dtype).to(DEV), kp, vp, table, step, 1.0, chunk=chunk)[-1]
                assert float((got.double().cpu() - want).abs().max()) < bar, (name, chunk, at_q, at)
            step = make_step([(i, at_q, 1) for i in range(n_seqs)])
            rows = q.expand(n_seqs, H, D).contiguous()
            for name in single:
                for splits in ((None,) if name == "attn_generic" else (1, None, 5)):
                    kw = {} if splits is None else {"n_splits": splits}
                    got = run_attention(name, rows.to(dtype).to(DEV), kp, vp, table, step, 1.0, chunk=chunk, **kw)
                    assert float((got.double().cpu() - want[None]).abs().max()) < bar, (name, splits, chunk, at_q, at)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D", [64, 128, 32, 144])
def test_chunked_and_windowed_prompts_of_unequal_sequences(dtype, D):
    """Sequences of other lengths and starts in one step, a padding sequence among them, chunks and
    windows shorter and longer than a page and than a block of query rows."""
    H, G = 4, 2
    lens = [(0, 300), (130, 1), (70, 140), (0, 65)]                       # (tokens before, rows of this step)
    T = 300
    k, v = rnd(T, G, D, seed=1, scale=D ** -0.25), rnd(T, G, D, seed=2)
    kp, vp, table = paged(k, v, None, 5, dtype)
    kd, vd = k.to(dtype).double(), v.to(dtype).double()
    seqs = [(i, st, n) for i, (st, n) in enumerate(lens)]
    seqs.insert(2, (-1, 0, 33))
    step = make_step(seqs)
    total = sum(n for _s, _st, n in seqs)
    q = rnd(total, H, D, seed=3, scale=2 * D ** -0.25).to(dtype)
    for kw, mask in [(dict(chunk=c), plain.chunk_mask(T, c)) for c in (1, 48, 64, 100, 129, 1000)] + \
                    [(dict(window=w), plain.window_mask(T, w)) for w in (1, 63, 128, 200)] + \
                    [(dict(window=40, chunk=90), plain.window_mask(T, 40) & plain.chunk_mask(T, 90))]:
        for name in attention_kernels(dtype, D)[0]:
            got = run_attention(name, q.to(DEV), kp, vp, table, step, 1.0, **kw).float().cpu()
            at = 0
            for slot, st, n in seqs:
                part = got[at:at + n]
                if slot < 0:
                    assert float(part.abs().max()) == 0.0
                else:
                    want = torch.stack([plain.masked_softmax_attention(
                        torch.cat([torch.zeros(st, D), q[at:at + n, h].float()]), kd[:st + n, h // 2],
                        vd[:st + n, h // 2], 1.0, mask[:st + n, :st + n])[st:] for h in range(H)], dim=1)
                    close(part, want, dtype, f"{name} {kw} sequence {slot}")
                at += n


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,Dv,Ds", [(1, 4, 64, 64), (70, 3, 20, 48), (9, 8, 128, 128), (5, 2, 300, 320), (33, 1, 7, 7), (4, 2, 512, 512)])
def test_the_difference_of_two_maps(dtype, T, H, Dv, Ds):
    from grout_b200.kernels import ops
    x = rnd(T, 2 * H, Ds, seed=1).to(dtype)
    lam, eps, mult = 0.83, 1e-3, 0.4
    d = x.double().view(T, H, 2, Ds)[..., :Dv]
    want = plain.over_rms(d[:, :, 0] - lam * d[:, :, 1], eps) * mult
    close(ops.diff_heads(x.to(DEV), Dv, lam, eps, mult), want.reshape(T, H * Dv), dtype)
    small = (x.double() * 1e-3).to(dtype)                       # below eps: the eps is inside the root
    d = small.double().view(T, H, 2, Ds)[..., :Dv]
    want = plain.over_rms(d[:, :, 0] - lam * d[:, :, 1], eps) * mult
    close(ops.diff_heads(small.to(DEV), Dv, lam, eps, mult), want.reshape(T, H * Dv), dtype)


# ------------------------------------------------------------------ the attention mixers over a paged cache
DIFF_SHAPES = [dict(heads=4, kv_heads=2, dim=16, vdim=32, chunk=7, dims=8, diff=0.3),
               dict(heads=2, kv_heads=1, dim=32, vdim=64, chunk=65, dims=32, diff=0.8),
               dict(heads=8, kv_heads=2, dim=64, vdim=128, chunk=96, dims=64, diff=0.5),
               dict(heads=3, kv_heads=3, dim=20, vdim=24, chunk=50, dims=4, diff=0.0),
               dict(heads=2, kv_heads=2, dim=16, vdim=80, chunk=None, dims=0, diff=0.6),
               dict(heads=20, kv_heads=1, dim=8, vdim=16, chunk=33, dims=8, diff=0.2)]


def walk_cuts(part, x, cuts, cache, view=0):
    """The rows of x through a mixer in steps of the given sizes, on a slot of its own, with another
    request holding pages in between; returns the results of all rows."""
    held = cache.open()
    cache.reserve(held, 70)
    slot = cache.open()
    outs, start = [], 0
    for n in cuts:
        cache.reserve(slot, n)
        cache.flush()
        y = part.forward(x[start:start + n].to(DEV), make_step([(slot, start, n)]), cache.view(view))
        outs.append((y.sum(0) if y.dim() == 3 else y).float().cpu())
        cache.advance(slot, n)
        start += n
    cache.close(held)
    cache.close(slot)                                             # the pages serve the next cut
    cache.check()
    return torch.cat(outs)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", DIFF_SHAPES)
def test_differential_attention_whole_in_portions_and_token_by_token(dtype, m):
    from grout_b200.cache import CacheLayout, SequenceCache
    from grout_b200.parts import PartSpec
    W, T, H, G, D, Dv = 48, 210, m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    w = {"q": rnd(2 * H * D, W, seed=1, scale=0.4), "k": rnd(2 * G * D, W, seed=2, scale=0.4),
         "v": rnd(G * Dv, W, seed=3, scale=0.5), "o": rnd(W, H * Dv, seed=4, scale=0.3)}
    w.update({n: rnd(D, seed=5 + i, scale=0.3) for i, n in enumerate(("lq1", "lk1", "lq2", "lk2"))})
    w = {k: t.to(dtype) for k, t in w.items()}
    x = rnd(T, W, seed=9).to(dtype)
    cfg = dict(heads=H, kv_heads=G, dim=D, vdim=Dv, scale=1.3 * D ** -0.5, diff=m["diff"])
    if m["chunk"]:
        cfg["mask"] = {"size": m["chunk"]}
    scaling = SCALINGS[4]
    if m["dims"]:
        cfg["rot"] = dict(base=900.0, dims=m["dims"], scaling=scaling)
    pw = {"m." + k: t for k, t in w.items()}
    run = lambda c, weights=pw: plain.differential_attention(x.double(), weights, "m.", c, list(range(T)), 1e-5)
    want = run(cfg)
    if m["chunk"] and m["chunk"] < 60:            # one more or one less position a chunk shows
        for dc in (-1, 1):
            off = run(dict(cfg, mask={"size": m["chunk"] + dc}))
            assert float((off - want).abs().max()) > 0.05 * float(want.abs().max())
    no_lq = dict(pw, **{"m.lq1": pw["m.lq1"] * 0})
    assert float((run(cfg, no_lq) - want).abs().max()) > 0.01 * float(want.abs().max())
    position = (PartSpec("rotary_half_split", dict(head_dim=D, theta=900.0, rot_dim=m["dims"], scaling=scaling))
                if m["dims"] else PartSpec("none", {}))
    part = make_part("mixer", "differential_attention", dtype, hidden=W, n_heads=H, n_kv_heads=G, head_dim=D,
                     v_head_dim=Dv, position=position, scale=1.3 * D ** -0.5, diff=m["diff"], norm_eps=1e-5,
                     chunk=m["chunk"])
    part.load({k: t.to(DEV) for k, t in w.items()})
    cache = SequenceCache(CacheLayout.from_specs([part.cache_spec()]), max_tokens=1024, max_slots=3,
                          max_seq_len=256, dtype=dtype, device=DEV)
    for cuts in ([T], [100] + [1] * 110, [63, 2, 64, 1, 70, 1, 1, 8], [2] * (T // 2), [1] * T):
        got = walk_cuts(part, x, cuts, cache)
        if dtype == torch.float32:
            close(got, want, dtype, str(cuts[:4]), scale=float(want.abs().max()))
        else:
            rows_close(got, want, str(cuts[:4]))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [dict(heads=4, kv_heads=2, dim=96, vdim=64, own=30, other=100, dims=96),
                               dict(heads=2, kv_heads=2, dim=64, vdim=64, own=130, other=5, dims=16),
                               dict(heads=4, kv_heads=1, dim=24, vdim=40, own=64, other=None, dims=24),
                               dict(heads=3, kv_heads=3, dim=32, vdim=16, own=None, other=1, dims=0)])
def test_a_layer_that_reads_another_layers_keys(dtype, m):
    """Queries, window and output projection of its own over the keys and values that another layer
    stored, whose window may be shorter (the pages stay for the reader) or longer."""
    from grout_b200.cache import CacheLayout, SequenceCache
    from grout_b200.parts import PartSpec
    W, T, H, G, D, Dv = 40, 230, m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    scaling = SCALINGS[0]
    position = (PartSpec("rotary_half_split", dict(head_dim=D, theta=900.0, rot_dim=m["dims"], scaling=scaling))
                if m["dims"] else PartSpec("none", {}))
    names = {"q": "q", "k": "k", "v": "v", "o": "o"}
    a, b = {}, {}
    for seed, w in ((1, a), (11, b)):
        w.update({"q": rnd(H * D, W, seed=seed, scale=0.4), "o": rnd(W, H * Dv, seed=seed + 1, scale=0.3)})
    a.update({"k": rnd(G * D, W, seed=3, scale=0.4), "v": rnd(G * Dv, W, seed=4, scale=0.5)})
    a, b = ({k: t.to(dtype) for k, t in w.items()} for w in (a, b))
    common = dict(hidden=W, n_heads=H, n_kv_heads=G, head_dim=D, v_head_dim=Dv, position=position, names=names)
    owner = make_part("mixer", "gqa_attention", dtype, scale=D ** -0.5, window=m["own"], reach=m["other"], **common)
    reader = make_part("mixer", "gqa_attention", dtype, scale=0.7 * D ** -0.5, window=m["other"], shares_kv=True, **common)
    owner.load({k: t.to(DEV) for k, t in a.items()})
    reader.load({k: t.to(DEV) for k, t in b.items()})
    assert reader.cache_spec() is None and "k" not in reader.param_specs()
    xa, xb = rnd(T, W, seed=5).to(dtype), rnd(T, W, seed=6).to(dtype)
    pos = list(range(T))
    cfg = lambda size, scale: dict(heads=H, kv_heads=G, dim=D, vdim=Dv, scale=scale,
                                   mask={"size": size} if size else None,
                                   rot=dict(base=900.0, dims=m["dims"], scaling=scaling) if m["dims"] else None)
    pa, pb = {"m." + k: t for k, t in a.items()}, {"m." + k: t for k, t in b.items()}
    stored = plain.window_keys_values(xa.double(), pa, "m.", cfg(m["own"], 1.0), pos)
    want_a = plain.window_attention(xa.double(), pa, "m.", cfg(m["own"], D ** -0.5), pos, stored)
    want_b = plain.window_attention(xb.double(), pb, "m.", cfg(m["other"], 0.7 * D ** -0.5), pos, stored)
    cache = SequenceCache(CacheLayout.from_specs([owner.cache_spec(), None]), max_tokens=1024, max_slots=3,
                          max_seq_len=256, dtype=dtype, device=DEV)
    for cuts in ([T], [150] + [1] * 80, [63, 2, 64, 1, 70, 1, 1, 28], [2] * (T // 2)):
        held, slot = cache.open(), cache.open()
        cache.reserve(held, 70)
        outs, start = ([], []), 0
        for n in cuts:
            cache.reserve(slot, n)
            cache.flush()
            step = make_step([(slot, start, n)])
            for part, x, out in ((owner, xa, outs[0]), (reader, xb, outs[1])):
                y = part.forward(x[start:start + n].to(DEV), step, cache.view(0))
                out.append((y.sum(0) if y.dim() == 3 else y).float().cpu())
            cache.advance(slot, n)
            start += n
        cache.close(held)
        cache.close(slot)
        for got, want, nm in ((torch.cat(outs[0]), want_a, "owner"), (torch.cat(outs[1]), want_b, "reader")):
            if dtype == torch.float32:
                close(got, want, dtype, f"{nm} {cuts[:3]}", scale=float(want.abs().max()))
            else:
                rows_close(got, want, f"{nm} {cuts[:3]}")
    cache.check()


# ------------------------------------------------------------------ lightning attention
def _light(heads, dim, vdim, lo=0.3, hi=0.999):
    return dict(heads=heads, dim=dim, vdim=vdim, decay=[lo + (hi - lo) * i / max(heads - 1, 1) for i in range(heads)])


def _light_weights(m, W, seed):
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    return {"q": rnd(H * dk, W, seed=seed, scale=0.4), "k": rnd(H * dk, W, seed=seed + 1, scale=0.4),
            "v": rnd(H * dv, W, seed=seed + 2, scale=0.4), "g": rnd(H * dv, W, seed=seed + 3, scale=0.4),
            "norm": 1 + rnd(H * dv, seed=seed + 4, scale=0.3), "o": torch.eye(H * dv)}


def _light_step(w, m, rows, state, seqs, dtype, max_rows="known"):
    from grout_b200.kernels import ops
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    wp = torch.cat([w[k] for k in ("q", "k", "v", "g")], 0).double()
    step = make_step(seqs)
    return ops.retention_forward(
        g32(rows.double() @ wp.T), state, torch.tensor(m["decay"], dtype=torch.float32, device=DEV), None, H=H,
        dk=dk, dv=dv, rot_dim=0, k_scale=1.0, norm_eps=1e-5, token_pos=step.token_pos, cu_q=step.cu_q,
        slots=step.slots, dtype=dtype, max_rows=step.max_q_len if max_rows == "known" else max_rows, silu=True,
        joint_norm=g32(w["norm"])).float().cpu()


def _light_run(w, m, xs, cuts, dtype):
    state = torch.zeros(3, m["heads"] * m["dim"] * m["vdim"], device=DEV)
    outs, start = [], 0
    for n in cuts:
        outs.append(_light_step(w, m, xs[start:start + n], state, [(1, start, n)], dtype))
        start += n
    return torch.cat(outs), state


def _light_plain(w, m, xs):
    return plain.lightning_attention(xs.double(), {"m." + k: v for k, v in w.items()}, "m.", m, 1e-5)


LIGHT_SHAPES = [_light(4, 16, 8), _light(3, 40, 20), _light(2, 64, 48), _light(1, 128, 16), _light(2, 30, 10),
                _light(1, 256, 40), _light(5, 8, 3), _light(2, 20, 300), _light(1, 1, 1), _light(2, 128, 128, lo=0.9)]


@pytest.mark.parametrize("m", LIGHT_SHAPES)
def test_lightning_attention_whole_in_portions_and_token_by_token(m):
    W, T = 24, 150
    w, xs = _light_weights(m, W, seed=3), rnd(T, W, seed=4)
    want = _light_plain(w, m, xs)
    whole, state = _light_run(w, m, xs, [T], torch.float32)
    close(whole, want, torch.float32, "whole")
    silu = lambda z: z * torch.sigmoid(z)
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    k, v = silu(xs.double() @ w["k"].double().T).view(T, H, dk), silu(xs.double() @ w["v"].double().T).view(T, H, dv)
    S = torch.stack([plain.fading_state_head(k[:, i], k[:, i], v[:, i], m["decay"][i])[1] for i in range(H)])
    close(state[1].view(H, dk, dv), S, torch.float32, "state", scale=float(S.abs().max()))
    assert float(state[[0, 2]].abs().max()) == 0.0
    for cuts in ([2] * 75, [1] * T, [1, 2, 3, 100, 44], [149, 1]):
        got, _ = _light_run(w, m, xs, cuts, torch.float32)
        close(got, whole, torch.float32, str(cuts[:4]))
    half, _ = _light_run(w, m, xs, [T], torch.bfloat16)
    close(half, want, torch.bfloat16, "bfloat16 output")


@pytest.mark.parametrize("m", [_light(3, 40, 20), _light(2, 64, 130, lo=0.9), _light(1, 128, 128, lo=0.97),
                               _light(2, 18, 30, lo=0.5, hi=0.9999), _light(3, 64, 64), _light(2, 64, 128, lo=0.99),
                               _light(2, 128, 64, lo=0.8, hi=1.0)])
def test_lightning_attention_long_sequences_go_chunk_by_chunk(m):
    """Long sequences beside short ones and a padding sequence, lengths at a chunk's edge, from states
    an earlier portion left; then single steps from the kept states; slots used again."""
    W, H, dk, dv = 24, m["heads"], m["dim"], m["vdim"]
    w = _light_weights(m, W, seed=21)
    lens, head = [256, 3, 257, 383, 1, 300], [0, 5, 2, 130, 0, 64]
    xs = [rnd(h + n + 2, W, seed=50 + i) for i, (h, n) in enumerate(zip(head, lens))]
    want = [_light_plain(w, m, x) for x in xs]
    kept = []
    for max_rows in ("known", None):                              # chunk by chunk, then row by row
        state = torch.full((len(lens) + 2, H * dk * dv), 7.0, device=DEV)
        state[1:len(lens) + 1].zero_()
        first = [(i + 1, 0, h) for i, h in enumerate(head) if h]
        _light_step(w, m, torch.cat([xs[s - 1][:h] for s, _, h in first]), state, first, torch.float32, None)
        seqs = [(i + 1, h, n) for i, (h, n) in enumerate(zip(head, lens))]
        rows = [x[h:h + n] for x, h, n in zip(xs, head, lens)]
        seqs.insert(3, (-1, 0, 260))
        rows.insert(3, rnd(260, W, seed=49))
        y = _light_step(w, m, torch.cat(rows), state, seqs, torch.float32, max_rows)
        at = 0
        for slot, h, n in seqs:
            if slot > 0:
                close(y[at:at + n], want[slot - 1][h:h + n], torch.float32, f"{max_rows}: {h} then {n} rows")
            at += n
        assert float((state[[0, len(lens) + 1]] - 7.0).abs().max()) == 0.0
        kept.append(state.clone())
        for j in (0, 1):                                          # two single steps, in another order, with padding
            order = [5, 0, 2, 1, 4, 3]
            y = _light_step(w, m, torch.cat([xs[i][head[i] + lens[i] + j][None] for i in order] + [rnd(1, W, seed=48)]),
                            state, [(i + 1, head[i] + lens[i] + j, 1) for i in order] + [(-1, 0, 1)], torch.float32)
            for r, i in enumerate(order):
                close(y[r], want[i][head[i] + lens[i] + j], torch.float32, f"single step {j} after {lens[i]}")
    close(kept[0], kept[1], torch.float32, "kept states", scale=float(kept[1].abs().max()))


def test_lightning_attention_reads_a_far_pair():
    """What was written 400 tokens ago under one key comes back under a slow decay when that key is
    asked for, and is gone under a fast one."""
    W = 32
    m = dict(heads=1, dim=16, vdim=8, decay=[0.999])
    w = {"q": torch.eye(16, W) * 4, "k": torch.eye(16, W) * 4, "v": torch.zeros(8, W), "g": torch.zeros(8, W),
         "norm": torch.ones(8), "o": torch.eye(8)}
    w["v"][:, 16:24] = torch.eye(8)
    w["g"][:, 24] = 1.0
    xs = torch.zeros(402, W)
    xs[:, 24] = 2.0
    xs[:, 3], xs[:, 16] = 0.02, 0.05                              # every token writes a little under key 3
    xs[0, 5], xs[0, 16:24] = 5.0, torch.arange(1.0, 9.0)          # the planted pair: key 5 -> value
    xs[401, 5] = 5.0                                              # the last token asks for key 5
    for decay, keeps in ((0.999, True), (0.9, False)):
        m["decay"] = [decay]
        got, _ = _light_run(w, m, xs, [300, 101, 1], torch.float32)
        close(got, _light_plain(w, m, xs), torch.float32, f"decay {decay}")
        x2 = xs.clone()
        x2[0, 16:24] = 0.0
        other, _ = _light_run(w, m, x2, [402], torch.float32)
        assert (float((got[401] - other[401]).abs().max()) > 0.1) == keeps, decay


# ------------------------------------------------------------------ routed experts
MOE_SHAPES = [dict(E=12, top=4, F=24, W=64, groups=(4, 2), scale=2.5, shared=40),
              dict(E=8, top=2, F=16, W=48, groups=(8, 3), scale=1.0, shared=16),      # one expert a group
              dict(E=6, top=6, F=20, W=36, groups=(3, 3), scale=0.7, shared=None),    # all of them
              dict(E=1, top=1, F=8, W=24, groups=None, scale=1.7, shared=72),
              dict(E=64, top=8, F=32, W=40, groups=(8, 2), scale=2.0, shared=24),
              dict(E=40, top=3, F=16, W=32, groups=None, scale=1.3, shared=None)]


def _moe(m, dtype, seed=0, correction=None):
    E, F, W = m["E"], m["F"], m["W"]
    w = {"router": rnd(E, W, seed=seed + 1, scale=0.6),
         "correction": rnd(E, seed=seed + 2, scale=0.6) - 0.9 if correction is None else correction}
    for e in range(E):
        w[f"e{e}.up"] = rnd(F, W, seed=seed + 10 + 2 * e, scale=0.3)
        w[f"e{e}.down"] = rnd(W, F, seed=seed + 11 + 2 * e, scale=0.3)
    if m["shared"]:
        w["shared.up"], w["shared.down"] = rnd(m["shared"], W, seed=seed + 3, scale=0.3), rnd(W, m["shared"], seed=seed + 4, scale=0.3)
    w = {k: v.to(dtype) for k, v in w.items()}
    g = m["groups"]
    part = make_part("feedforward", "routed_experts", dtype, hidden=W, intermediate=F, n_experts=E, top=m["top"],
                     score_fn="sigmoid", gated=False, n_groups=g[0] if g else 1, keep_groups=g[1] if g else 1,
                     group_score="top2", normalize=True, weight_scale=m["scale"], shared_intermediate=m["shared"])
    part.load({k: v.to(DEV) for k, v in w.items()})
    mlp = {"router": {"top": m["top"], "scale": m["scale"]}}
    if g:
        mlp["router"]["groups"] = {"count": g[0], "keep": g[1]}
    if m["shared"]:
        mlp["shared"] = {"ff": m["shared"]}
    return part, w, mlp


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [1, 5, 33, 70, 600])
@pytest.mark.parametrize("m", MOE_SHAPES)
def test_ungated_experts_groups_and_the_shared_expert(monkeypatch, dtype, T, m):
    """Choice scores that are mostly negative, so that a dropped group that were left at zero would win;
    few rows and many (the products' kernels differ)."""
    part, w, mlp = _moe(m, dtype)
    x = rnd(T, m["W"], seed=5).to(dtype)
    pw = {"m." + k: v for k, v in w.items()}
    want = plain.experts_ff(x.double(), pw, "m.", mlp)
    from grout_b200.kernels import ops
    for products in ("auto", "tiles", "pair") if dtype == torch.bfloat16 else ("auto",):
        monkeypatch.setattr(ops, "MOE_PRODUCTS", products)
        got = part.forward(x.to(DEV), None)
        assert got.dtype == torch.float32 and got.shape[0] >= m["top"] + (1 if m["shared"] else 0)
        got = got.sum(0).double().cpu()
        if dtype == torch.float32:
            close(got, want, dtype, scale=float(want.abs().max()))
        else:      # a near tie between two experts may fall the other way after rounding: most rows agree
            rows = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
            assert float(rows.median()) < 0.02 and float((rows < 0.06).double().mean()) > 0.9, products
        if T == 70:     # a token's result does not depend on the rows around it
            alone = part.forward(x[11:12].to(DEV), None).sum(0).double().cpu()
            close(alone[0], got[11], dtype, products, scale=float(want.abs().max()) / (1 if dtype == torch.float32 else 8))
    ops.check_kernel_errors()


@pytest.mark.parametrize("T", [1, 12, 64, 130, 700])
@pytest.mark.parametrize("shape", [(6, 2, 24, 64, 0, 0), (3, 3, 200, 96, 2, 1), (1, 1, 136, 40, 0, 0), (40, 4, 72, 264, 0, 1)])
def test_experts_on_pairs_of_SMs_and_in_tiles_agree(T, shape):
    """The grouped product on pairs of SMs against the tile kernels, gated and ungated, with a clamp, an
    offset, outputs that hand the input on and weights on the input; experts without rows, with fewer
    than a tile's and with more; widths that end inside a tile."""
    from grout_b200.kernels import ops
    E, top, F, W, identity, weigh = shape
    bf = torch.bfloat16
    x = rnd(T, W, seed=1).to(bf).to(DEV)
    router = g32(rnd(E + identity, W, seed=2, scale=0.5))
    if E > 5:
        router[4] = -router[0]                              # (an expert that is chosen rarely)
        router[5] = -1.0e3 * router[1].abs() * x[0].float().sign()
    wg, wu, wd = (rnd(*s, seed=3 + i, scale=0.3).to(bf).to(DEV) for i, s in enumerate(((E, F, W), (E, F, W), (E, W, F))))
    shared = (rnd(88, W, seed=7, scale=0.3).to(bf).to(DEV), rnd(W, 88, seed=8, scale=0.3).to(bf).to(DEV))
    for gate in (wg, None):
        for sh in ((None, shared) if gate is None else (None,)):
            outs = []
            for products in ("tiles", "pair"):
                ops.MOE_PRODUCTS = products
                try:
                    outs.append(ops.moe_forward(x, router, None, gate, wu, wd, top=top, n_identity=identity,
                                                limit=1.5 if gate is not None else math.inf, slope=1.3,
                                                weigh_input=bool(weigh), up_offset=0.5, shared=sh))
                finally:
                    ops.MOE_PRODUCTS = "auto"
            assert outs[0].shape[0] == top + (1 if sh else 0)
            scale = float(outs[0].abs().max())
            assert scale > 0.1 and not torch.isnan(outs[1]).any()
            # the inner activations are rounded to bfloat16 from sums taken in another order
            assert float((outs[0] - outs[1]).abs().max()) < 0.02 * scale
            assert float((outs[0] - outs[1]).pow(2).mean().sqrt()) < 0.002 * scale
    ops.check_kernel_errors()


def test_the_choice_goes_by_corrected_scores_and_the_weights_do_not():
    """Corrections that turn the choice round, groups that win by their second expert, ties."""
    from grout_b200.kernels import ops
    E, W, top = 8, 16, 2
    x = torch.zeros(3, W)
    x[0, 0] = x[1, 1] = x[2, 2] = 1.0
    router = torch.zeros(E, W)
    router[:, 0] = torch.tensor([3.0, -3.0, 1.0, 0.9, 0.0, 0.0, -1.0, -1.0])     # group 0 has the largest, group 1 the best two
    router[:, 1] = 0.5                                                           # all equal
    router[:, 2] = torch.arange(8.0)
    corr = torch.zeros(E)
    run = lambda c, **kw: ops.moe_forward(x.to(DEV), router.to(DEV), c.to(DEV), None, torch.zeros(E, 4, W, device=DEV),
                                          torch.zeros(E, W, 4, device=DEV), top=top, score_fn="sigmoid",
                                          want_choice=True, **kw)
    groups = dict(n_groups=4, keep_groups=1)
    _o, ids, wts = run(corr, group_top2=True, normalize=True, weight_scale=2.5, **groups)
    assert ids.cpu().tolist() == [[2, 3], [0, 1], [7, 6]]
    s = torch.sigmoid(router.double() @ x.double().T).T
    for t, chosen in enumerate([[2, 3], [0, 1], [7, 6]]):
        close(wts[t], s[t, chosen] / s[t, chosen].sum() * 2.5, torch.float32)
    _o, ids, _w = run(corr, group_top2=False, **groups)                          # by its largest alone: group 0
    assert ids.cpu()[0].tolist() == [0, 1]
    corr = torch.tensor([-9.0, -9.0, -9.0, -9.0, -2.0, -1.0, -9.0, -9.0])        # every choice score is negative
    _o, ids, wts = run(corr, group_top2=True, normalize=True, **groups)
    assert ids.cpu().tolist() == [[5, 4], [5, 4], [5, 4]]
    close(wts[2], s[2, [5, 4]] / s[2, [5, 4]].sum(), torch.float32)              # the weights: scores without it
    for t in range(3):
        chosen, p = plain.route(s[t], corr.double(), {"top": top, "scale": 1.0, "groups": {"count": 4, "keep": 1}})
        assert chosen == ids[t].tolist()
        close(wts[t], p, torch.float32)


def test_a_result_goes_into_the_tensor_it_is_given():
    """The products that leave their 32-bit sums behind another kernel's: every kernel a linear layer
    can take, few rows and many, widths that are and are not multiples of eight."""
    from grout_b200.parts.base import ProductChoice
    from grout_b200.parts.linear import Linear
    for K, N, dtype in ((64, 48, torch.bfloat16), (2048, 256, torch.bfloat16), (36, 20, torch.bfloat16), (40, 24, torch.float32)):
        w, want_w = rnd(N, K, seed=1, scale=K ** -0.5).to(dtype), None
        for choice in (ProductChoice(), ProductChoice(decode="skinny", prefill="tc"), ProductChoice(prefill="pair")):
            lin = Linear(w.to(DEV), choice)
            for M in (1, 9, 64, 65, 300):
                x = rnd(M, K, seed=M).to(dtype)
                S = lin.n_parts(M)
                stack = torch.full((S + 2, M, N), 5.0, device=DEV)
                y = lin(x.to(DEV), into=stack[1:1 + S])
                assert y.data_ptr() == stack[1].data_ptr()
                close(stack[1:1 + S].sum(0), x.double() @ w.double().T, torch.float32, f"{K} {N} {M} {choice}")
                assert float((stack[[0, S + 1]] - 5.0).abs().max()) == 0.0
