"""Plain Keralix decoder: whole sequences, no cache, one function per mechanism.

Keralix is a pre-norm decoder on several residual streams.  The streams X_1 .. X_s all
start as E[token] * c.  A sublayer F (a mixer or a feed-forward, behind an RMS norm N) reads
a weighted sum of them and its result goes back into all of them, while the streams are
mixed with one another ("hyper-connections"):

    y = F(N(sum_s a_s X_s));    X_t <- sum_s M[s, t] X_s + b_t y

The model's last norm reads the plain sum of the streams.  A layer's mixer is one of

* windowed attention with short causal convolutions behind the query and key projections,
  values that are the convolved keys in front of their rotation, and capped scores;
* attention without positions whose queries and keys both come from latent vectors, with a
  learned sink in the softmax's denominator and an elementwise gate on the heads' output;
* a delta rule whose state fades by one factor per key channel and token.

The feed-forward, where a layer has one, is silu-gated.  All arithmetic is float64 on the
CPU.  Inputs are a dict ``name -> tensor`` with the checkpoint's tensor names and the raw
``config.json`` dict.  Nothing here is shared with the product package.
"""
from __future__ import annotations

import math

import torch

DT = torch.float64
UNIT_EPS = 1e-6           # under the root that makes queries and keys unit vectors


def over_rms(x, eps):
    x = x.to(DT)
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + float(eps))


def rms_norm(x, w, eps):
    return over_rms(x, eps) * w.to(DT)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def unit(x):
    x = x.to(DT)
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + UNIT_EPS)


# -- streams ----------------------------------------------------------------
def read_streams(X, a):
    """sum_s a_s X_s for X [streams, T, W]."""
    u = torch.zeros_like(X[0])
    for s in range(X.shape[0]):
        u = u + float(a[s]) * X[s]
    return u


def write_streams(X, M, b, y):
    """New stream t: sum_s M[s, t] X_s + b_t y, every one from the old streams."""
    n = X.shape[0]
    return torch.stack([sum(float(M[s, t]) * X[s] for s in range(n)) + float(b[t]) * y for t in range(n)])


# -- shared by the mixers ---------------------------------------------------
def short_conv(x, taps_w):
    """x [T, C], taps_w [C, taps]: channel c of row t becomes
    sum_j taps_w[c, j] x[t - taps + 1 + j, c], rows in front of the sequence being zeros."""
    x, w = x.to(DT), taps_w.to(DT)
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            src = t - taps + 1 + j
            if src >= 0:
                y[t] += w[:, j] * x[src]
    return y


def rotate_halves(x, positions, base, dims):
    """x [T, heads, D]: of the first ``dims`` elements, i turns with i + dims/2 by
    p * base^(-2i/dims)."""
    x = x.to(DT)
    half = dims // 2
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=DT)
    a = torch.as_tensor(positions, dtype=DT)[:, None] * f
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v, rest = x[..., :half], x[..., half:dims], x[..., dims:]
    return torch.cat([u * c - v * s, v * c + u * s, rest], dim=-1)


def sees_window(T, size):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    d = i - j
    return (d >= 0) & (d < int(size)) if size else d >= 0


def softmax_attention(q, k, v, scale, mask, cap=None, sink=None):
    """One head: q [T, D], k [T, D], v [T, Dv], mask [T, T] of visible pairs.  ``sink`` is a
    logit that stands in the denominator alone."""
    s = (q.to(DT) @ k.to(DT).T) * float(scale)
    if cap:
        s = float(cap) * torch.tanh(s / float(cap))
    s = s.masked_fill(~mask, -math.inf)
    if sink is not None:
        extra = torch.full((s.shape[0], 1), float(sink), dtype=DT)
        return torch.softmax(torch.cat([s, extra], dim=1), dim=1)[:, :-1] @ v.to(DT)
    return torch.softmax(s, dim=1) @ v.to(DT)


# -- mixers -----------------------------------------------------------------
def convolved_attention(h, w, p, m, positions):
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    h, t = h.to(DT), lambda n: w[p + n].to(DT)
    T = h.shape[0]
    q = short_conv(h @ t("q").T + t("q.b"), t("q.conv")).view(T, H, D)
    k = short_conv(h @ t("k").T + t("k.b"), t("k.conv")).view(T, G, D)
    v = k
    rot = m.get("rot")
    if rot and rot["dims"]:
        q, k = (rotate_halves(x, positions, rot["base"], rot["dims"]) for x in (q, k))
    mask = sees_window(T, m["mask"]["size"] if m.get("mask") else None)
    heads = [softmax_attention(q[:, i], k[:, i // (H // G)], v[:, i // (H // G)], m["scale"], mask,
                               cap=m.get("softcap")) for i in range(H)]
    return torch.cat(heads, dim=-1) @ t("o").T


def latent_attention(h, w, p, m, eps):
    H, D, Dv = m["heads"], m["dim"], m["vdim"]
    h, t = h.to(DT), lambda n: w[p + n].to(DT)
    T = h.shape[0]
    q = (rms_norm(h @ t("dq").T, t("dq.norm"), eps) @ t("uq").T).view(T, H, D)
    c = rms_norm(h @ t("dkv").T, t("dkv.norm"), eps)
    k, v = (c @ t("uk").T).view(T, H, D), (c @ t("uv").T).view(T, H, Dv)
    mask = sees_window(T, None)
    heads = [softmax_attention(q[:, i], k[:, i], v[:, i], m["scale"], mask, sink=t("sink")[i]) for i in range(H)]
    return (torch.cat(heads, dim=-1) * torch.sigmoid(h @ t("g").T)) @ t("o").T


def channel_decays(h, w, p, H, D):
    """[T, H, D]: exp(-exp(A_log) softplus(low-rank + dt_bias)), A_log one number a head."""
    h, t = h.to(DT), lambda n: w[p + n].to(DT)
    x = softplus((h @ t("a1").T) @ t("a2").T + t("dt_bias")).view(-1, H, D)
    return torch.exp(-torch.exp(t("A_log"))[None, :, None] * x)


def delta_head(q, k, v, beta, g, S=None):
    """One head.  q, k, g [T, D]; v [T, Dv]; beta [T].  The rows of S [D, Dv] fade by g, the
    key's current value is moved towards v by beta, and q reads afterwards."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=DT) if S is None else S.to(DT)
    out = []
    for i in range(k.shape[0]):
        S = g[i].to(DT)[:, None] * S
        u = beta[i] * (v[i].to(DT) - S.T @ k[i].to(DT))
        S = S + torch.outer(k[i].to(DT), u)
        out.append(S.T @ q[i].to(DT))
    return torch.stack(out), S


def delta_mixer(h, w, p, m, eps):
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    h, t = h.to(DT), lambda n: w[p + n].to(DT)
    T = h.shape[0]
    q = unit(silu(short_conv(h @ t("q").T, t("q.conv"))).view(T, G, D)) * D ** -0.5
    k = unit(silu(short_conv(h @ t("k").T, t("k.conv"))).view(T, G, D))
    v = silu(short_conv(h @ t("v").T, t("v.conv"))).view(T, H, Dv)
    beta = torch.sigmoid(h @ t("b").T)
    g = channel_decays(h, w, p, H, D)
    gate = torch.sigmoid((h @ t("g1").T) @ t("g2").T).view(T, H, Dv)
    heads = []
    for i in range(H):
        j = i // (H // G)
        o, _S = delta_head(q[:, j], k[:, j], v[:, i], beta[:, i], g[:, i])
        heads.append(rms_norm(o, t("norm"), eps) * gate[:, i])
    return torch.cat(heads, dim=-1) @ t("o").T


def feed_forward(h, w, p):
    h, t = h.to(DT), lambda n: w[p + n].to(DT)
    return (silu(h @ t("gate").T) * (h @ t("up").T)) @ t("down").T


def mixer(kind, h, w, p, m, eps, positions):
    if kind == "attention":
        return convolved_attention(h, w, p, m, positions)
    if kind == "latent_attention":
        return latent_attention(h, w, p, m, eps)
    return delta_mixer(h, w, p, m, eps)


# -- the model --------------------------------------------------------------
def forward(tokens, w, cfg, return_layers=False):
    """Logits [T, vocab] of one sequence from its first token (and, when asked, the sum of
    the streams behind every layer)."""
    eps, n = cfg["norm"]["eps"], cfg["streams"]
    table = w["embed"].to(DT)
    x = table[torch.as_tensor(tokens)] * float(cfg["embedding"]["scale"])
    X = torch.stack([x] * n)
    positions = torch.arange(len(tokens))
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        subs = [lambda z: mixer(layer["type"], z, w, p + "mix.", layer["mixer"], eps, positions)]
        if layer.get("mlp") is not None:
            subs.append(lambda z: feed_forward(z, w, p + "mlp."))
        for k, sub in enumerate(subs, 1):
            hc = f"{p}hc{k}."
            y = sub(rms_norm(read_streams(X, w[hc + "in"]), w[f"{p}norm{k}"], eps))
            X = write_streams(X, w[hc + "mix"], w[hc + "out"], y)
        after.append(X.sum(dim=0))
    out = rms_norm(X.sum(dim=0), w["final.norm"], eps) @ table.T
    return (out, torch.stack(after)) if return_layers else out


def logits(w, cfg, tokens, rows=None):
    out = forward(list(tokens), w, cfg)
    return out if rows is None else out[list(rows)]


def greedy_generate(w, cfg, prompt, n_new, stop_ids=()):
    """The plain loop: the whole sequence is recomputed for every new token."""
    seq, made = list(prompt), []
    for _ in range(n_new):
        tok = int(torch.argmax(forward(seq, w, cfg)[-1]))
        if tok in stop_ids:          # a stop token ends the request and is not part of its output
            break
        made.append(tok)
        seq.append(tok)
    return made
