"""Plain Kakotar decoder: whole sequences, no cache, one function per mechanism.

Kakotar is a pre-norm decoder, x <- x + M(N1(x)); x <- x + F(N2(x)) (the second line
only where the layer has an F).  Its norm N is a dynamic tanh, which looks at single
elements only; it has no statistics of a row.  A layer's mixer M is one of

* lightning attention: a matrix-valued state per head that fades by a fixed factor a
  token, read without a softmax; queries, keys and values pass a silu, the heads'
  read-outs are normalised together and gated,
* softmax attention over a window of the last tokens with rotated queries and keys,
  the rotation's frequencies stretched by the YaRN rule; a layer may read the keys and
  values that another layer has stored, with queries of its own,
* differential attention within fixed chunks of the sequence: two attention maps a head
  over the same values, the second subtracted from the first times a learned number,
  the rotation's frequencies stretched band by band.

F is a mixture of small ungated squared-relu experts with one more that runs for every
token: sigmoid scores, a correction that takes part in the choice only, a choice within
the best groups of experts, weights that add up to a constant.

All arithmetic is float64 on the CPU.  Inputs are a dict ``name -> tensor`` with the
checkpoint's tensor names and the raw ``config.json`` dict.  Nothing here is shared with
the product package.
"""
from __future__ import annotations

import math

import torch

DT = torch.float64


def silu(z):
    return z * torch.sigmoid(z)


def dynamic_tanh(x, w, name):
    """tanh(alpha x) * weight + bias; alpha is one number."""
    alpha = w[name + ".alpha"].to(DT).reshape(())
    return torch.tanh(alpha * x.to(DT)) * w[name].to(DT) + w[name + ".b"].to(DT)


def over_rms(x, eps):
    x = x.to(DT)
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + float(eps))


# ---------------------------------------------------------------- rotation
def plain_frequencies(base, dims):
    return [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]


def yarn_frequencies(base, dims, factor, original, fast, slow):
    """Elements that turn often within the original length keep their frequency, those that
    turn rarely have it divided, with a straight ramp over the elements between."""
    def element_of(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(element_of(fast)), 0)
    hi = min(math.ceil(element_of(slow)), dims - 1)
    out = []
    for i, f in enumerate(plain_frequencies(base, dims)):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out


def yarn_amplitude(factor):
    return 0.1 * math.log(factor) + 1.0


def banded_frequencies(base, dims, factor, low, high, original):
    """Short wavelengths stay, long ones are divided, those between are mixed."""
    out = []
    for f in plain_frequencies(base, dims):
        wave = 2.0 * math.pi / f
        if wave < original / high:
            out.append(f)
        elif wave > original / low:
            out.append(f / factor)
        else:
            s = (original / wave - low) / (high - low)
            out.append((1.0 - s) * f / factor + s * f)
    return out


def rotation_of(rot):
    """(frequencies, amplitude) of a configuration's 'rot'."""
    if not rot or not rot["dims"]:
        return [], 1.0
    s = rot.get("scaling")
    if not s:
        return plain_frequencies(rot["base"], rot["dims"]), 1.0
    if "fast" in s:
        return (yarn_frequencies(rot["base"], rot["dims"], s["factor"], s["original"], s["fast"], s["slow"]),
                yarn_amplitude(s["factor"]))
    return banded_frequencies(rot["base"], rot["dims"], s["factor"], s["low"], s["high"], s["original"]), 1.0


def rotate(x, positions, frequencies, amplitude=1.0):
    """x [T, ..., D]: element i of the first 2 n goes with element i + n, n frequencies."""
    n = len(frequencies)
    if n == 0:
        return x
    x = x.to(DT).clone()
    ang = torch.as_tensor(positions, dtype=DT)[:, None] * torch.tensor(frequencies, dtype=DT)[None, :]
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [n]
    c, s = (torch.cos(ang) * amplitude).view(shape), (torch.sin(ang) * amplitude).view(shape)
    u, v = x[..., :n].clone(), x[..., n:2 * n].clone()
    x[..., :n] = u * c - v * s
    x[..., n:2 * n] = v * c + u * s
    return x


# ---------------------------------------------------------------- attention
def window_mask(T, size):
    """[T, T]: row i sees column j when 0 <= i - j < size (None: no bound)."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) if size is None else (d >= 0) & (d < int(size))


def chunk_mask(T, size):
    """[T, T]: row i sees column j <= i of its own chunk of ``size`` positions."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) if size is None else (j <= i) & (i // int(size) == j // int(size))


def masked_softmax_attention(q, k, v, scale, mask):
    """One head: q [T, D], k [T, D], v [T, Dv]."""
    s = (q.to(DT) @ k.to(DT).T) * float(scale)
    return torch.softmax(s.masked_fill(~mask, -math.inf), dim=-1) @ v.to(DT)


def window_keys_values(h, w, p, m, positions):
    """What a windowed attention layer stores: rotated keys [T, G, dim], values [T, G, vdim]."""
    T, G = h.shape[0], m["kv_heads"]
    f, amp = rotation_of(m.get("rot"))
    k = rotate((h @ w[p + "k"].to(DT).T).view(T, G, m["dim"]), positions, f, amp)
    return k, (h @ w[p + "v"].to(DT).T).view(T, G, m["vdim"])


def window_attention(h, w, p, m, positions, stored):
    """``stored``: the (keys, values) that the layer reads, its own or another layer's."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    f, amp = rotation_of(m.get("rot"))
    q = rotate((h @ w[p + "q"].to(DT).T).view(T, H, m["dim"]), positions, f, amp)
    k, v = stored
    mask = window_mask(T, m["mask"]["size"] if m.get("mask") else None)
    heads = [masked_softmax_attention(q[:, i], k[:, i // (H // G)], v[:, i // (H // G)], m["scale"], mask)
             for i in range(H)]
    return torch.cat(heads, dim=-1) @ w[p + "o"].to(DT).T


def difference_factor(w, p, diff):
    """The one number a layer subtracts its second maps with."""
    s = lambda a, b: float((w[p + a].to(DT) * w[p + b].to(DT)).sum())
    return math.exp(s("lq1", "lk1")) - math.exp(s("lq2", "lk2")) + float(diff)


def differential_attention(h, w, p, m, positions, eps):
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    f, amp = rotation_of(m.get("rot"))
    q = rotate((h @ w[p + "q"].to(DT).T).view(T, H, 2, D), positions, f, amp)
    k = rotate((h @ w[p + "k"].to(DT).T).view(T, G, 2, D), positions, f, amp)
    v = (h @ w[p + "v"].to(DT).T).view(T, G, m["vdim"])
    mask = chunk_mask(T, m["mask"]["size"] if m.get("mask") else None)
    lam, diff = difference_factor(w, p, m["diff"]), float(m["diff"])
    heads = []
    for i in range(H):
        g = i // (H // G)
        a1, a2 = (masked_softmax_attention(q[:, i, n], k[:, g, n], v[:, g], m["scale"], mask) for n in (0, 1))
        heads.append(over_rms(a1 - lam * a2, eps) * (1.0 - diff))
    return torch.cat(heads, dim=-1) @ w[p + "o"].to(DT).T


# ---------------------------------------------------------------- lightning attention
def fading_state_head(q, k, v, decay, S=None):
    """One head: S <- decay S + k v^T; o = S^T q.  Returns (read-outs, last S)."""
    q, k, v = q.to(DT), k.to(DT), v.to(DT)
    S = torch.zeros(k.shape[1], v.shape[1], dtype=DT) if S is None else S.to(DT)
    out = []
    for t in range(q.shape[0]):
        S = float(decay) * S + torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out), S


def lightning_attention(h, w, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q = silu(h @ w[p + "q"].to(DT).T).view(T, H, m["dim"])
    k = silu(h @ w[p + "k"].to(DT).T).view(T, H, m["dim"])
    v = silu(h @ w[p + "v"].to(DT).T).view(T, H, m["vdim"])
    o = torch.cat([fading_state_head(q[:, i], k[:, i], v[:, i], m["decay"][i])[0] for i in range(H)], dim=-1)
    o = over_rms(o, eps) * w[p + "norm"].to(DT) * torch.sigmoid(h @ w[p + "g"].to(DT).T)
    return o @ w[p + "o"].to(DT).T


# ---------------------------------------------------------------- feed-forward
def relu_squared_ff(h, w, p):
    return torch.relu(h @ w[p + "up"].to(DT).T) ** 2 @ w[p + "down"].to(DT).T


def route(scores, correction, router):
    """For one token: (chosen experts, their weights).  The choice is by score + correction,
    within the groups whose two best such sums add up to most; the weights are the scores
    alone, scaled to add up to ``scale``."""
    E, c = scores.shape[0], scores + correction
    g = router.get("groups")
    if g:
        per = E // g["count"]
        value = [float(torch.sort(c[i * per:(i + 1) * per], descending=True).values[:2].sum())
                 for i in range(g["count"])]
        best = sorted(range(g["count"]), key=lambda i: -value[i])[:g["keep"]]
        allowed = [e for i in sorted(best) for e in range(i * per, (i + 1) * per)]
    else:
        allowed = list(range(E))
    chosen = sorted(allowed, key=lambda e: -float(c[e]))[:router["top"]]
    s = scores[chosen]
    return chosen, s / (s.sum() + 1e-20) * float(router["scale"])


def experts_ff(h, w, p, mlp):
    scores = torch.sigmoid(h @ w[p + "router"].to(DT).T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, wt = route(scores[t], w[p + "correction"].to(DT), mlp["router"])
        for e, a in zip(chosen, wt):
            out[t] += a * relu_squared_ff(h[t:t + 1], w, f"{p}e{e}.")[0]
    if mlp.get("shared"):
        out = out + relu_squared_ff(h, w, p + "shared.")
    return out


# ---------------------------------------------------------------- the model
def forward(tokens, w, cfg, return_layers=False):
    """Logits [T, vocab] of one sequence from its first token."""
    eps = cfg["norm"]["eps"]
    positions = list(range(len(tokens)))
    x = w["embed"].to(DT)[torch.as_tensor(list(tokens), dtype=torch.long)]
    stored, after = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        h = dynamic_tanh(x, w, f"l{i}.norm1")
        if layer["type"] == "lightning":
            y = lightning_attention(h, w, p, m, eps)
        elif layer["type"] == "attention_2":
            y = differential_attention(h, w, p, m, positions, eps)
        else:
            src = m.get("kv_from")
            if src is None:
                stored[i] = window_keys_values(h, w, p, m, positions)
            y = window_attention(h, w, p, m, positions, stored[i if src is None else src])
        x = x + y
        if layer.get("mlp") is not None:
            x = x + experts_ff(dynamic_tanh(x, w, f"l{i}.norm2"), w, f"l{i}.mlp.", layer["mlp"])
        after.append(x)
    out = dynamic_tanh(x, w, "final.norm") @ w["head"].to(DT).T
    return (out, torch.stack(after)) if return_layers else out


def logits(w, cfg, tokens, rows=None):
    out = forward(tokens, w, cfg)
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
