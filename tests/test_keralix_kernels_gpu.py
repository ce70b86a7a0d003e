"""Each mechanism that the Keralix design brought, alone, against the plain implementation's
function for it: residual streams that are mixed at a sublayer boundary, attention behind
biases and short convolutions (planted window edges, the sequence's first tokens, cuts inside
the convolution's reach), query latents and sinks in latent attention, and the delta rule with
a decay per key channel (step, scan and chunk by chunk; strong decays; far keys; slots used
again; padding rows)."""
import math

import pytest
import torch

from plain import keralix as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
BAR = {torch.float32: 3e-5, torch.bfloat16: 0.02}
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


def close(got, want, dtype, what="", bar=None):
    """Largest error against the largest value."""
    got, want = got.detach().double().cpu(), want.detach().double().cpu()
    assert got.shape == want.shape, (what, got.shape, want.shape)
    assert bool(torch.isfinite(got).all()), what
    err, top = (got - want).abs(), float(want.abs().max())
    assert float(err.max()) <= (bar or BAR[dtype]) * max(top, 1e-3), \
        f"{what}: max err {err.max().item():.3g} of {top:.3g} at {int(err.argmax())}"


def apart(got, want, wrong, rows, what=""):
    """The result is nearer to what is right than to what a fault would give, by far."""
    got, want, wrong = (t.detach().double().cpu()[rows] for t in (got, want, wrong))
    rms = lambda t: float(t.pow(2).mean().sqrt())
    assert rms(got - want) < 0.25 * rms(wrong - want), f"{what}: {rms(got - want):.3g} against {rms(wrong - want):.3g}"


def rnd(*shape, seed=0, scale=1.0, dtype=torch.float32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def make_step(seqs):
    """The fields of a step that the kernels read, for sequences given as (slot, start, n)."""
    from grout_b200.engine.batch import make_context
    return make_context([(s, st, [0] * n) for s, st, n in seqs], None, DEV)


def build(kind, weights, dtype, **args):
    from grout_b200.parts import BuildContext, PartSpec, build_part
    part = build_part("mixer", PartSpec(kind, args), BuildContext(dtype, torch.device(DEV)))
    part.load({k: v.to(DEV) for k, v in weights.items()})
    return part


def cache_for(part, dtype, slots=4):
    from grout_b200.cache import CacheLayout, SequenceCache
    return SequenceCache(CacheLayout.from_specs([part.cache_spec()]), max_tokens=2048, max_slots=slots,
                         max_seq_len=512, dtype=dtype, device=DEV)


def feed(part, cache, xs, schedule):
    """``xs``: rows of each sequence; ``schedule``: steps, each a dict sequence -> rows it brings.
    Sequences open when they first bring rows and close when theirs are used up."""
    slots, at, outs = {}, [0] * len(xs), [[] for _ in xs]
    for bring in schedule:
        seqs, rows = [], []
        for i, n in bring.items():
            if i not in slots:
                slots[i] = cache.open()
            cache.reserve(slots[i], n)
            seqs.append((slots[i], at[i], n))
            rows.append(xs[i][at[i]:at[i] + n])
        cache.flush()
        y = part.forward(torch.cat(rows).to(DEV), make_step(seqs), cache.view(0))
        y = (y.sum(0) if y.dim() == 3 else y).float().cpu()
        o = 0
        for i, n in bring.items():
            outs[i].append(y[o:o + n])
            o, at[i] = o + n, at[i] + n
            cache.advance(slots[i], n)
            if at[i] == len(xs[i]):
                cache.close(slots.pop(i))
    assert at == [len(x) for x in xs]
    return [torch.cat(o) for o in outs]


def cuts_of(sizes):
    return [{0: n} for n in sizes]


def in_layer(w, dtype):
    """Weights as the part gets them and as the plain function does (the same rounded values)."""
    w = {k: v.to(dtype) for k, v in w.items()}
    return w, {"m." + k: v for k, v in w.items()}


# ------------------------------------------------------------------ residual streams
@BOTH
@pytest.mark.parametrize("sizes", [(1, 24, 5), (2, 100, 3), (3, 1024, 70), (4, 288, 9), (4, 2560, 130), (5, 512, 8),
                                   (8, 96, 4), (8, 1024, 2), (11, 36, 6), (4, 37, 3)])
def test_streams_mixed_read_and_normalised_in_one_kernel(dtype, sizes):
    from grout_b200.kernels import ops
    S, N, T = sizes
    X, d = rnd(S, T, N, seed=1, scale=2.0), rnd(T, N, seed=2).to(dtype)
    M, b, a = rnd(S, S, seed=3), rnd(S, seed=4), rnd(S, seed=5)
    nw = 1 + rnd(N, seed=6, scale=0.2)
    g = lambda t: t.to(DEV)
    kw = dict(streams=S, dtype=dtype, mix=g(M), write=g(b))
    want = plain.write_streams(X.double(), M, b, d.double())
    want_y = plain.rms_norm(plain.read_streams(want, a), nw, 1e-5)
    stack = g(X)
    res, y = ops.hyper_norm(stack, g(d), read=g(a), norm_w=g(nw), eps=1e-5, **kw)
    assert res.data_ptr() == stack.data_ptr()                       # in place
    close(res, want, torch.float32, "streams")
    close(y, want_y, dtype, "normalised")
    parts = torch.stack([d.float() * f for f in (0.25, 0.5, 0.125, 0.0625, 0.0625)]).contiguous()
    res, y = ops.hyper_norm(g(X), g(parts), read=g(a), norm_w=g(nw), eps=1e-5, **kw)
    close(res, want, torch.float32, "streams from partial sums")
    close(y, want_y, dtype, "normalised, from partial sums")
    # streams that are still equal; the first sublayer, which has nothing to put back
    same = plain.write_streams(torch.stack([X[0]] * S).double(), M, b, d.double())
    res, y = ops.hyper_norm(g(X[0]), g(d), read=g(a), norm_w=g(nw), eps=1e-5, **kw)
    close(res, same, torch.float32, "streams from equal ones")
    first = g(X[0])
    res, y = ops.hyper_norm(first, None, streams=S, dtype=dtype, read=g(a), norm_w=g(nw), eps=1e-5)
    assert res is first and torch.equal(first.cpu(), X[0])
    close(y, plain.rms_norm(X[0].double() * float(a.double().sum()), nw, 1e-5), dtype, "first sublayer")
    # the last norm: the streams' sum, gathered rows, nothing kept
    rows = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32)
    stack = g(X)
    _res, y = ops.hyper_norm(stack, g(d), rows=g(rows), norm_w=g(nw), eps=1e-5, **kw)
    assert torch.equal(stack.cpu(), X)
    close(y, plain.rms_norm(want.sum(0)[rows.long()], nw, 1e-5), dtype, "last norm")
    _res, y = ops.hyper_norm(g(X), g(d), read=g(a), **kw)
    close(y, plain.read_streams(want, a), dtype, "without a norm")


def test_norms_without_a_kernel_for_streams_resolve_them():
    from grout_b200.parts import BuildContext, HyperConnected, PartSpec, build_part
    S, T, N = 3, 6, 40
    X, d = rnd(S, T, N, seed=1), rnd(T, N, seed=2)
    M, b, a = rnd(S, S, seed=3), rnd(S, seed=4), rnd(S, seed=5)
    want = plain.write_streams(X.double(), M, b, d.double())
    u = plain.read_streams(want, a)
    norm = build_part("norm", PartSpec("layernorm", dict(dim=N, eps=1e-5)), BuildContext(torch.float32, torch.device(DEV)))
    norm.load({"weight": torch.ones(N, device=DEV), "bias": torch.zeros(N, device=DEV)})
    g = lambda t: t.to(DEV)
    res, y = norm.add_norm(g(X), HyperConnected(S, g(d), g(M), g(b), g(a)))
    close(res, want, torch.float32)
    c = u - u.mean(-1, keepdim=True)
    close(y, c / torch.sqrt((c * c).mean(-1, keepdim=True) + 1e-5), torch.float32)
    rows = torch.tensor([4, 1], dtype=torch.int32, device=DEV)
    _r, y = norm.add_norm(g(X), HyperConnected(S, g(d), g(M), g(b)), rows=rows)
    u = want.sum(0)[[4, 1]]
    c = u - u.mean(-1, keepdim=True)
    close(y, c / torch.sqrt((c * c).mean(-1, keepdim=True) + 1e-5), torch.float32)


# ------------------------------------------------------------------ attention behind convolutions
def _conv_weights(m, W, seed, sharp=1.0):
    H, G, D, taps = m["heads"], m["kv_heads"], m["dim"], m["conv"]
    return {"q": rnd(H * D, W, seed=seed, scale=sharp / W ** 0.5), "k": rnd(G * D, W, seed=seed + 1, scale=sharp / W ** 0.5),
            "q.b": rnd(H * D, seed=seed + 2, scale=0.5), "k.b": rnd(G * D, seed=seed + 3, scale=0.5),
            "q.conv": rnd(H * D, taps, seed=seed + 4, scale=1.2 * taps ** -0.5),
            "k.conv": rnd(G * D, taps, seed=seed + 5, scale=1.2 * taps ** -0.5), "o": rnd(W, H * D, seed=seed + 6, scale=(H * D) ** -0.5)}


def _conv_part(m, W, w, dtype):
    from grout_b200.parts import PartSpec
    rot, mask = m.get("rot"), m.get("mask")
    position = (PartSpec("rotary_half_split", dict(head_dim=m["dim"], theta=rot["base"], rot_dim=rot["dims"],
                                                   exact_table=True)) if rot else PartSpec("none", {}))
    return build("gqa_attention", w, dtype, hidden=W, n_heads=m["heads"], n_kv_heads=m["kv_heads"], head_dim=m["dim"],
                 position=position, scale=m["scale"], window=mask["size"] if mask else None, softcap=m.get("softcap"),
                 values_are_keys=True, qk_bias=True, conv_taps=m["conv"],
                 names={"q": "q", "k": "k", "o": "o", "q_bias": "q.b", "k_bias": "k.b", "q_conv": "q.conv",
                        "k_conv": "k.conv"})


def _conv(H, G, D, taps, window, cap, dims, base=1e4):
    return dict(heads=H, kv_heads=G, dim=D, conv=taps, scale=D ** -0.5, softcap=cap,
                mask={"size": window} if window else None, rot={"base": base, "dims": dims} if dims else None)


CONV_SHAPES = [_conv(6, 2, 48, 3, 17, 20.0, 48), _conv(6, 3, 64, 4, 64, None, 32), _conv(2, 1, 128, 2, 65, 5.0, 128),
               _conv(3, 3, 40, 5, 63, 30.0, 16), _conv(4, 1, 24, 1, None, 8.0, 0), _conv(2, 2, 20, 12, 130, None, 20),
               _conv(5, 5, 17, 3, 2, 15.0, 6)]


@BOTH
@pytest.mark.parametrize("m", CONV_SHAPES)
def test_attention_behind_convolutions_in_every_cut(dtype, m):
    """A prompt whole, token by token, in portions down to two rows; windows just inside and
    just outside; pages and slots that were another request's."""
    W, T = 56, 150
    w, pw = in_layer(_conv_weights(m, W, seed=20, sharp=3.0), dtype)
    x = rnd(T, W, seed=41).to(dtype)
    pos = torch.arange(T)
    want = plain.convolved_attention(x, pw, "m.", m, pos)
    size = m["mask"]["size"] if m["mask"] else 0
    wrong = [plain.convolved_attention(x, pw, "m.", dict(m, mask={"size": n}), pos) for n in (size - 1, size + 1) if size]
    part = _conv_part(m, W, w, dtype)
    cache = cache_for(part, dtype)
    for cuts in ([T], [1] * T, [2] * (T // 2), [66, 1, 1, 5, 64, 3, 10], [7, 8, 9, 1, 125], [3, T - 3]):
        got, = feed(part, cache, [x], cuts_of(cuts))
        close(got, want, dtype, f"cuts {cuts[:8]}")
        for other in wrong:
            apart(got, want, other, slice(size + 1, None), f"window, cuts {cuts[:8]}")
        cache.check()


@BOTH
def test_attention_behind_convolutions_in_mixed_batches(dtype):
    """Requests of unequal lengths together and alone; one-token and many-token rows in one step."""
    m, W = _conv(6, 2, 32, 4, 30, 20.0, 24), 40
    w, pw = in_layer(_conv_weights(m, W, seed=3, sharp=3.0), dtype)
    xs = [rnd(n, W, seed=50 + n).to(dtype) for n in (1, 75, 3, 34)]
    part = _conv_part(m, W, w, dtype)
    cache = cache_for(part, dtype)
    schedules = ([{0: 1, 1: 75, 2: 3, 3: 34}],
                 [{1: 70, 3: 30}, {1: 1, 2: 1, 3: 1}, {3: 1, 1: 1, 2: 1}, {2: 1, 1: 3, 3: 2, 0: 1}],
                 [{2: 2, 1: 9}, {1: 8, 2: 1, 3: 17}, {0: 1, 3: 17, 1: 58}])
    want = [plain.convolved_attention(x, pw, "m.", m, torch.arange(len(x))) for x in xs]
    for schedule in schedules:
        for i, got in enumerate(feed(part, cache, xs, schedule)):
            close(got, want[i], dtype, f"request {i}")


def test_zeros_and_not_biases_lie_in_front_of_a_sequence():
    """With projections of zero every input of the convolution is its bias: the first rows see
    fewer taps, whatever the slot held before."""
    m, W, T = _conv(2, 1, 16, 3, None, None, 0), 16, 6
    w = {k: v.float() for k, v in _conv_weights(m, W, seed=9).items()}
    w["q"].zero_(), w["k"].zero_()
    x = rnd(T, W, seed=1)
    part = _conv_part(m, W, w, torch.float32)
    cache = cache_for(part, torch.float32, slots=1)
    other = rnd(5, W, seed=2)
    for cuts in ([T], [1] * T, [2, 2, 2]):
        feed(part, cache, [other], cuts_of([5]))                    # the slot's former holder
        got, = feed(part, cache, [x], cuts_of(cuts))
        close(got, plain.convolved_attention(x, {"m." + k: v for k, v in w.items()}, "m.", m, torch.arange(T)),
              torch.float32)
    kb, kc = w["k.b"].double(), w["k.conv"].double()
    first, steady = kb * kc[:, 2], kb * kc.sum(1)
    assert float((first - steady).abs().max()) > 0.1                # (and the two differ)


@BOTH
@pytest.mark.parametrize("D,rows", [(32, 1), (20, 70)])
def test_convolved_queries_and_keys_with_values_of_their_own(dtype, D, rows):
    """The kernel with neighbouring pairs, values from the projection and partial sums of it."""
    from grout_b200.kernels import ops
    from grout_b200.parts.position import scaled_inverse_frequencies
    nq, nkv, Dv, taps, page, Ds, start = 4, 2, 12, 3, 64, 32, 60
    Cc = (nq + nkv) * D
    width = Cc + nkv * Dv
    proj = rnd(start + rows, width, seed=1)
    bias, cw = rnd(Cc, seed=2), rnd(Cc, taps, seed=3)
    dims = D - D % 4
    inv = torch.tensor(scaled_inverse_frequencies(dims, 1e4, None), dtype=torch.float32)
    kp, vp = (torch.zeros(4, nkv, page, Ds, dtype=dtype, device=DEV) for _ in range(2))
    table = torch.tensor([[9, 9, 9], [2, 0, 3]], dtype=torch.int32, device=DEV)
    tail = torch.full((3, (taps - 1) * Cc), 7.0, device=DEV)
    tail[1] = 0
    outs = []
    for a, b in ((0, start), (start, start + rows)):
        p = proj[a:b]
        parts = torch.stack([p * 0.5, p * 0.25, p * 0.25]).contiguous().to(DEV)
        outs.append(ops.qk_conv(parts, nq, nkv, D, step=make_step([(1, a, b - a)]), block_table=table, k_pages=kp,
                                v_pages=vp, page=page, taps=taps, bias=bias.to(DEV), conv_w=cw.to(DEV), tail=tail,
                                v_dim=Dv, inv_freq=inv.to(DEV), rot_dim=dims, interleaved=True, rot_scale=1.5))
    q = torch.cat(outs)
    u = proj[:, :Cc].double() + bias.double()
    c = plain.short_conv(u, cw).view(-1, nq + nkv, D)
    ang = torch.arange(start + rows, dtype=torch.float64)[:, None] * inv.double()
    cs, sn = 1.5 * torch.cos(ang)[:, None], 1.5 * torch.sin(ang)[:, None]
    e, o = c[..., 0:dims:2].clone(), c[..., 1:dims:2].clone()
    c[..., 0:dims:2], c[..., 1:dims:2] = e * cs - o * sn, o * cs + e * sn
    close(q[..., :D], c[:, :nq], dtype, "queries")
    assert not q[..., D:].any()
    where = [(int(table[1, t // page]), t % page) for t in range(start + rows)]
    close(torch.stack([kp[pg, :, r, :D] for pg, r in where]), c[:, nq:], dtype, "keys")
    close(torch.stack([vp[pg, :, r, :Dv] for pg, r in where]), proj[:, Cc:].view(-1, nkv, Dv), dtype, "values")
    close(tail[1].view(taps - 1, Cc), u[-(taps - 1):], torch.float32, "kept inputs")
    assert bool((tail[0] == 7).all()) and bool((tail[2] == 7).all())


# ------------------------------------------------------------------ latent attention
def _lat_weights(m, W, seed, sharp):
    H, D, Dv, Rq, R = m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"]
    n = lambda *s, k, sc: rnd(*s, seed=seed + k, scale=sc * s[-1] ** -0.5)
    return {"dq": n(Rq, W, k=0, sc=1.0), "dq.norm": 1 + rnd(Rq, seed=seed + 1, scale=0.2),
            "uq": n(H * D, Rq, k=2, sc=sharp), "dkv": n(R, W, k=3, sc=1.0),
            "dkv.norm": 1 + rnd(R, seed=seed + 4, scale=0.2), "uk": n(H * D, R, k=5, sc=sharp),
            "uv": n(H * Dv, R, k=6, sc=1.0), "sink": torch.linspace(-2.0, 4.0, H), "g": n(H * Dv, W, k=7, sc=2.0),
            "o": n(W, H * Dv, k=8, sc=1.0)}


def _lat(H, D, Dv, Rq, R, scale=None):
    return dict(heads=H, dim=D, vdim=Dv, q_rank=Rq, kv_rank=R, scale=scale or D ** -0.5)


@BOTH
@pytest.mark.parametrize("m", [_lat(5, 24, 40, 88, 128), _lat(3, 24, 16, 20, 40), _lat(20, 16, 24, 36, 64), _lat(2, 128, 32, 64, 150),
                               _lat(2, 8, 8, 8, 8, 0.6), _lat(17, 16, 16, 33, 24)])
def test_latent_queries_and_sinks_in_every_cut(dtype, m):
    from grout_b200.parts import PartSpec
    W, T, eps = 48, 140, 1e-3
    w, pw = in_layer(_lat_weights(m, W, seed=70, sharp=1.5), dtype)
    x = rnd(T, W, seed=71).to(dtype)
    want = plain.latent_attention(x, pw, "m.", m, eps)
    # a sink that is left out, or scaled with the scores, would show
    wrong = [plain.latent_attention(x, dict(pw, **{"m.sink": sink}), "m.", m, eps)
             for sink in (torch.full((m["heads"],), -1e30), w["sink"].float() * m["scale"])]
    part = build("latent_attention", w, dtype, hidden=W, n_heads=m["heads"], head_dim=m["dim"], rot_dim=0,
                 v_head_dim=m["vdim"], kv_rank=m["kv_rank"], q_rank=m["q_rank"], position=PartSpec("none", {}),
                 scale=m["scale"], norm_eps=eps, sinks=True)
    cache = cache_for(part, dtype)
    for cuts in ([T], [1] * T, [65, 2, 1, 1, 64, 3, 4], [2] * 70):
        got, = feed(part, cache, [x], cuts_of(cuts))
        close(got, want, dtype, f"cuts {cuts[:8]}")
        for other in wrong:
            apart(got, want, other, slice(0, 20), "sinks")
    xs = [x[:70], x[30:33], x[5:6]]
    for got, xi in zip(feed(part, cache, xs, [{0: 60, 1: 2}, {0: 1, 1: 1, 2: 1}, {0: 9}]), xs):
        close(got, plain.latent_attention(xi, pw, "m.", m, eps), dtype, "batch")


@BOTH
def test_a_far_key_among_hundreds_is_found(dtype):
    """One key's score stands out, hundreds of rows and many pages back: its value comes through."""
    from grout_b200.parts import PartSpec
    m, W, T, far, eps = _lat(2, 16, 16, 16, 32), 32, 400, 3, 1e-5
    w, pw = in_layer(_lat_weights(m, W, seed=5, sharp=4.0), dtype)
    x = rnd(T, W, seed=6)
    d = {k: v.double() for k, v in w.items()}
    # row 3 is made so that its latent is what the last row's first head asks for
    q = plain.rms_norm(x[T - 1].to(dtype).double() @ d["dq"].T, d["dq.norm"], eps) @ d["uq"][:16].T
    x[far] = (torch.linalg.solve(d["dkv"], (q @ d["uk"][:16]) / d["dkv.norm"])).float()
    x = x.to(dtype)
    want = plain.latent_attention(x, pw, "m.", m, eps)
    gone = plain.latent_attention(torch.cat([x[:far], x[far + 1:]]), pw, "m.", m, eps)
    part = build("latent_attention", w, dtype, hidden=W, n_heads=2, head_dim=16, rot_dim=0, v_head_dim=16, kv_rank=32,
                 q_rank=16, position=PartSpec("none", {}), scale=m["scale"], norm_eps=eps, sinks=True)
    cache = cache_for(part, dtype)
    for cuts in ([T], [T - 1, 1], [100, 299, 1]):
        got, = feed(part, cache, [x], cuts_of(cuts))
        close(got, want, dtype, f"cuts {cuts}", bar=None if dtype == torch.float32 else 0.05)   # (sharp scores)
        apart(got[-1:], want[-1:], gone[-1:], slice(None), "the far key")


@BOTH
def test_query_latents_beside_a_rotated_part(dtype):
    """The combination that this design leaves out: expanded queries with a rotated part."""
    from grout_b200.parts import PartSpec
    H, dn, dr, dv, Rq, R, W, T, eps = 3, 16, 8, 12, 24, 40, 36, 80, 1e-5
    w = _lat_weights(_lat(H, dn + dr, dv, Rq, R), W, seed=11, sharp=1.5)
    w["uk"], w["dkv"] = rnd(H * dn, R, seed=12, scale=1.5 * R ** -0.5), rnd(R + dr, W, seed=13, scale=W ** -0.5)
    w, _ = in_layer(w, dtype)
    x = rnd(T, W, seed=14).to(dtype)
    d = {k: v.double() for k, v in w.items()}
    turn = lambda t: _neighbours(t, 1e4)
    q = (plain.rms_norm(x.double() @ d["dq"].T, d["dq.norm"], eps) @ d["uq"].T).view(T, H, dn + dr)
    down = x.double() @ d["dkv"].T
    c, kr = plain.rms_norm(down[:, :R], d["dkv.norm"], eps), turn(down[:, None, R:])[:, 0]
    qr = turn(q[..., dn:])
    mask = plain.sees_window(T, None)
    heads = []
    for i in range(H):
        k = torch.cat([c @ d["uk"][i * dn:(i + 1) * dn].T, kr], -1)
        heads.append(plain.softmax_attention(torch.cat([q[:, i, :dn], qr[:, i]], -1), k, c @ d["uv"][i * dv:(i + 1) * dv].T,
                                             0.2, mask, sink=d["sink"][i]))
    want = (torch.cat(heads, -1) * torch.sigmoid(x.double() @ d["g"].T)) @ d["o"].T
    part = build("latent_attention", w, dtype, hidden=W, n_heads=H, head_dim=dn, rot_dim=dr, v_head_dim=dv, kv_rank=R,
                 q_rank=Rq, position=PartSpec("rotary_interleaved", dict(head_dim=dr, theta=1e4, rot_dim=dr,
                                                                         exact_table=True)),
                 scale=0.2, norm_eps=eps, sinks=True)
    cache = cache_for(part, dtype)
    for cuts in ([T], [70] + [1] * 10):
        got, = feed(part, cache, [x], cuts_of(cuts))
        close(got, want, dtype, f"cuts {cuts[:3]}")


def _neighbours(x, base):
    n = x.shape[-1]
    f = torch.tensor([base ** (-2.0 * i / n) for i in range(n // 2)], dtype=torch.float64)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None, None] * f
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a)], -1).flatten(-2)


# ------------------------------------------------------------------ the delta rule, a decay per channel
def _delta(H, G, D, Dv, taps, ra=10, rg=6):
    return dict(heads=H, kv_heads=G, dim=D, vdim=Dv, conv=taps, ra=ra, rg=rg)


def _delta_weights(m, W, seed, decay=0.0):
    """``decay``: added to A_log; heads go from slow to fast decays."""
    H, G, D, Dv, taps, ra, rg = (m[k] for k in ("heads", "kv_heads", "dim", "vdim", "conv", "ra", "rg"))
    n = lambda *s, k, sc=1.0: rnd(*s, seed=seed + k, scale=sc * s[-1] ** -0.5)
    return {"q": n(G * D, W, k=0), "k": n(G * D, W, k=1), "v": n(H * Dv, W, k=2, sc=1.5), "b": n(H, W, k=3, sc=2.0),
            "q.conv": n(G * D, taps, k=4), "k.conv": n(G * D, taps, k=5), "v.conv": n(H * Dv, taps, k=6),
            "A_log": torch.linspace(-5.0, 1.0, H) + decay, "a1": n(ra, W, k=7), "a2": n(H * D, ra, k=8, sc=2.0),
            "dt_bias": rnd(H * D, seed=seed + 9), "g1": n(rg, W, k=10), "g2": n(H * Dv, rg, k=11, sc=2.0),
            "norm": 1 + rnd(Dv, seed=seed + 12, scale=0.2), "o": n(W, H * Dv, k=13)}


def _delta_part(m, W, w, dtype, eps=1e-5):
    return build("channel_delta", w, dtype, hidden=W, n_heads=m["heads"], n_kv_heads=m["kv_heads"], key_dim=m["dim"],
                 value_dim=m["vdim"], conv_taps=m["conv"], norm_eps=eps)


# heads of 64 and 128 and odd ones, several heads on one key, one tap, more taps than rows of a step
DELTA_SHAPES = [_delta(3, 3, 64, 48, 3), _delta(4, 2, 128, 128, 4, 24, 24), _delta(3, 1, 20, 36, 2, 5, 3), _delta(2, 2, 16, 10, 1),
                _delta(2, 1, 33, 17, 5), _delta(1, 1, 96, 160, 10), _delta(2, 2, 200, 24, 3)]


@BOTH
@pytest.mark.parametrize("m", DELTA_SHAPES)
def test_channel_delta_in_every_cut(dtype, m):
    W, T = 40, 170
    w, pw = in_layer(_delta_weights(m, W, seed=90), dtype)
    x = rnd(T, W, seed=91).to(dtype)
    want = plain.delta_mixer(x, pw, "m.", m, 1e-5)
    part = _delta_part(m, W, w, dtype)
    cache = cache_for(part, dtype)
    for cuts in ([T], [1] * T, [2] * 85, [64, 63, 3, 33, 7], [65, 1, 1, 96, 7], [32, 31, 107]):
        got, = feed(part, cache, [x], cuts_of(cuts))
        close(got, want, dtype, f"cuts {cuts[:6]}")


@BOTH
def test_channel_delta_in_mixed_batches(dtype):
    m, W = _delta(4, 2, 32, 24, 4), 32
    w, pw = in_layer(_delta_weights(m, W, seed=7), dtype)
    xs = [rnd(n, W, seed=60 + n).to(dtype) for n in (2, 140, 1, 97)]
    want = [plain.delta_mixer(x, pw, "m.", m, 1e-5) for x in xs]
    part = _delta_part(m, W, w, dtype)
    cache = cache_for(part, dtype)
    for schedule in ([{0: 2, 1: 140, 2: 1, 3: 97}], [{1: 64, 0: 1}, {1: 1, 0: 1, 3: 1}, {1: 75, 2: 1, 3: 96}],
                     [{3: 33, 1: 31}, {1: 96, 3: 64}, {1: 13}, {0: 2, 2: 1}]):
        for i, got in enumerate(feed(part, cache, xs, schedule)):
            close(got, want[i], dtype, f"request {i}")


@pytest.mark.parametrize("decay", [3.0, 6.0, -6.0])
def test_channel_delta_with_extreme_decays(decay):
    """Decays from "gone within a row" (their products underflow inside a chunk) to "kept for
    ever", channels of one head apart from one another; nothing overflows in any cut."""
    m, W, T = _delta(3, 3, 64, 32, 3, 16, 8), 24, 200
    w, pw = in_layer(_delta_weights(m, W, seed=17, decay=decay), torch.float32)
    w["a2"] *= 4.0
    x = rnd(T, W, seed=18)
    want = plain.delta_mixer(x, pw, "m.", m, 1e-5)
    part = _delta_part(m, W, w, torch.float32)
    cache = cache_for(part, torch.float32)
    for cuts in ([T], [1] * T, [100, 100], [40] * 5):
        got, = feed(part, cache, [x], cuts_of(cuts))
        close(got, want, torch.float32, f"cuts {cuts[:3]}", bar=1e-4)


def test_channel_delta_reads_a_far_value():
    """A value that one row writes under a key of its own is read 300 rows later through channels
    that keep, and is gone through channels that fade."""
    from grout_b200.kernels import ops
    H = G = 1
    dk, dv, T = 8, 4, 320
    q, k = torch.zeros(T, dk), torch.zeros(T, dk)
    v = rnd(T, dv, seed=1)
    k[:, :4] = rnd(T, 4, seed=2)                    # other rows write elsewhere
    k[5] = torch.tensor([0, 0, 0, 0, 1.0, 0, 0, 0])
    q[T - 1] = k[5]
    for keeps in (True, False):
        z = torch.full((T, dk), -12.0)              # softplus(z): next to no decay
        if not keeps:
            z[:, 4] = 1.0
        big = lambda t: torch.where(t != 0, t, torch.zeros_like(t))
        proj = torch.cat([big(q), big(k), v, torch.full((T, 1), 30.0), torch.zeros(T, 8)], 1)
        conv = torch.ones(2 * dk + dv, 1)
        wide = torch.cat([z, torch.full((T, dv), 30.0)], 1)
        silu = lambda t: t * torch.sigmoid(t)
        o, _ = plain.delta_head(plain.unit(silu(q.double())) * dk ** -0.5, plain.unit(silu(k.double())), silu(v.double()),
                                torch.ones(T, dtype=torch.float64), torch.exp(-plain.softplus(z.double())))
        want = plain.over_rms(o, 1e-12)
        step = make_step([(0, 0, T)])
        sizes = dict(H=1, G=1, dk=dk, dv=dv, taps=1, token_seq=step.token_seq, cu_q=step.cu_q, slots=step.slots,
                     dtype=torch.float32)
        g = lambda t: t.float().contiguous().to(DEV)
        for rows in (T, 2):                         # chunk by chunk, and row by row
            state = torch.zeros(2, H * dk * dv, device=DEV)
            p = g(proj)
            prep, low = ops.channel_delta_prepare(p, state, g(conv), n_low=8, unit_eps=1e-6, **sizes)
            y = ops.channel_delta_run(p, prep, low, g(wide), state, g(conv), g(torch.zeros(1)), g(torch.zeros(dk)),
                                      g(torch.ones(dv)), norm_eps=1e-12, max_rows=rows, **sizes)
            if keeps:
                close(y[-1], want[-1], torch.float32, "the far value", bar=1e-3)
            size = float(o[-1].norm() / silu(v[5].double()).norm())
            assert (size > 0.3) if keeps else (size < 1e-6)
            # the state in 32-bit
            close(state[0].view(dv, dk).T, plain.delta_head(torch.zeros(T, dk), plain.unit(silu(k.double())), silu(v.double()),
                                                            torch.ones(T, dtype=torch.float64),
                                                            torch.exp(-plain.softplus(z.double())))[1],
                  torch.float32, "state", bar=1e-4)


def test_channel_delta_padding_rows_store_nothing():
    m, W = _delta(2, 1, 16, 12, 3), 24
    w, pw = in_layer(_delta_weights(m, W, seed=27), torch.float32)
    part = _delta_part(m, W, w, torch.float32)
    cache = cache_for(part, torch.float32)
    slot = cache.open()
    cache.reserve(slot, 90)
    cache.flush()
    x = rnd(90, W, seed=28)
    view = cache.view(0)
    for pad in (1, 80):                              # a step of single rows, a step of many
        before = view.state.clone()
        part.forward(rnd(pad, W, seed=29).to(DEV), make_step([(-1, 0, pad)]), view)
        assert torch.equal(view.state, before)
    y = part.forward(torch.cat([x, x[:7]]).to(DEV), make_step([(slot, 0, 90), (-1, 0, 7)]), view)
    y = (y.sum(0) if y.dim() == 3 else y)
    close(y[:90], plain.delta_mixer(x, pw, "m.", m, 1e-5), torch.float32)
