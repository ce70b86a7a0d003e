#!/usr/bin/env python3
"""Decode and prefill throughput of the engine at Qwen3-4B layer sizes with
random weights on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W]

A "step" is one decode step of the whole batch (default 8 sequences that each
hold a 2,048-token prompt, context 4096).  ``value`` is decoded tokens per
second timed on the device with CUDA events over exactly K steps; ``regions``
cuts the same K steps into five consecutive regions (an event between them) and
gives the median and the quartiles of their times per step, in the manner of
the reference's repetitions (benchmarks/src/bin/grout_bench.rs:218-252);
``e2e`` is the same through ``Engine.generate`` with host token lists in and
out.  The line also carries the 2,048-token prefill, the decode step's HBM
roofline and decode at batch 1 and 64.  Every decode step reads the 8 GB of
weights, far more than the 126 MB L2, so nothing is flushed between timed steps.

    python bench.py --size 8b|32b      the same run at the other sizes of the workload list
    python bench.py --ops [--size S] [--batch B]
                                       a table of every kernel of one prompt step and of
                                       decode steps (launched one by one, an event pair
                                       around each): calls, time, GB/s, TFLOP/s, fractions
    python bench.py --requests S       the reference's request grid
    python bench.py --designs [--design suvazen|sonalorn|zutazen|mananex|kakotar|keralix] [--design-sizes 1b,4b,8b] [--batch B] [--design-ops]
                                       prefill and decode throughput of the Suvazen (or Sonalorn)
                                       design beside the Qwen3 decoder at equal layer sizes (random weights), and
                                       with --design-ops the per-kernel tables of both
"""
import argparse
import json
import os
import statistics
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

QWEN3_4B = dict(architectures=["Qwen3ForCausalLM"], model_type="qwen3", vocab_size=151936,
                hidden_size=2560, intermediate_size=9728, num_hidden_layers=36,
                num_attention_heads=32, num_key_value_heads=8, head_dim=128, rope_theta=1000000.0,
                rms_norm_eps=1e-6, max_position_embeddings=40960, tie_word_embeddings=True,
                use_sliding_window=False, eos_token_id=151645)
# The other two model sizes of the workload list, for --requests (layer sizes only; the
# default run and its contract stay with the 4B sizes).
SIZES = {
    "4b": QWEN3_4B,
    "8b": dict(QWEN3_4B, hidden_size=4096, intermediate_size=12288, tie_word_embeddings=False),
    "32b": dict(QWEN3_4B, hidden_size=5120, intermediate_size=25600, num_hidden_layers=64,
                num_attention_heads=64, tie_word_embeddings=False),
}
# What the reference publishes for Qwen3-32B on a B200 (fp16, batch 1, its own engine):
# request_gen_tps = generated tokens / seconds of the whole request, and one prefill time
# (benchmarks/RESULTS.md:29-31, 45-47, 53-55).  (prompt tokens, generated tokens) -> figure.
PUBLISHED_32B = {(18, 36): 79.6, (18, 128): 79.9, (18, 512): 80.1, (128, 36): 79.0, (512, 36): 75.3,
                 (2048, 36): 61.4, (8192, 36): 37.2}
PUBLISHED_32B_PREFILL_MS = {8192: 513.78}
CONTEXT = 4096
PROMPT = 2048
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0}
SETTLE_S = 0.5      # idle between a batch's prompts and its decode steps (see decode_run)
REGIONS = 5


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        try:
            with open(path) as fh:
                p = json.load(fh)
            return {"hbm_gbs": float(p["hbm_gbs"]), "bf16_tflops": float(p["bf16_tflops"]),
                    "bf16_tflops_sustained": float(p.get("bf16_tflops_sustained", p["bf16_tflops"])),
                    "source": "measured"}
        except Exception:
            pass
    return dict(FALLBACK_PEAKS, source="fallback")


class ClockSampler:
    """nvidia-smi clocks and throttle reasons every 200 ms while the timed region runs."""
    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,"
             "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
             "clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.rows, self.proc = [], None

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits",
                 "-lms", "200"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.rows.append([c.strip() for c in line.split(",")])

    def stop(self):
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        time.sleep(0.25)
        self.proc.terminate()
        sm = [int(r[0]) for r in self.rows if r and r[0].isdigit()]
        mx = [int(r[1]) for r in self.rows if len(r) > 1 and r[1].isdigit()]
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = sorted({n for r in self.rows if len(r) >= 6
                          for n, v in zip(names, r[2:6]) if v.lower().startswith("active")})
        return {"sm_mhz": int(statistics.median(sm)) if sm else None,
                "sm_max_mhz": max(mx) if mx else None, "reasons": reasons}


def weight_bytes(cfg, layers):
    H, D = cfg["hidden_size"], cfg["head_dim"]
    nq, nkv, I, V = cfg["num_attention_heads"], cfg["num_key_value_heads"], cfg["intermediate_size"], cfg["vocab_size"]
    per_layer = (nq + 2 * nkv) * D * H + nq * D * H + 3 * H * I + 2 * H + 2 * D
    return 2 * (layers * per_layer + V * H + H)          # bf16; the head reads the table once


def kv_bytes_per_token(cfg, layers):
    return layers * 2 * cfg["num_key_value_heads"] * cfg["head_dim"] * 2


def prefill_flops(cfg, layers, T):
    H, D = cfg["hidden_size"], cfg["head_dim"]
    nq, nkv, I, V = cfg["num_attention_heads"], cfg["num_key_value_heads"], cfg["intermediate_size"], cfg["vocab_size"]
    linear = 2 * T * ((nq + 2 * nkv) * D * H + nq * D * H + 3 * H * I)
    attn = 2 * 2 * nq * D * T * (T + 1) // 2
    return layers * (linear + attn) + 2 * V * H


def run_requests(size: str, reps: int) -> int:
    """The reference's own request grid (one sequence: prompt of P tokens, T tokens generated,
    EOS ignored) through ``Engine.generate`` with random weights of the named size and random
    token ids: generated tokens per second of the whole request, host tokens in and out; the
    median of ``reps`` requests after two that are discarded, half a second apart."""
    import torch
    from grout_b200.engine import Engine
    cfg = SIZES[size]
    eng = Engine.random(cfg, 0, dtype="bfloat16", max_tokens=8192 + 576, max_batch=1,
                        max_seq_len=8192 + 512 + 64)
    g = torch.Generator().manual_seed(1)

    def prompt(n):
        return torch.randint(0, cfg["vocab_size"], (n,), generator=g).tolist()

    cells = []
    for pp, tg in sorted(PUBLISHED_32B):
        runs = []
        for i in range(reps + 2):
            time.sleep(0.5)
            o = eng.generate([prompt(pp)], tg, ignore_eos=True)[0]
            if i >= 2:
                runs.append((o.generated_tokens / o.total_elapsed, o.prompt_elapsed * 1e3,
                             o.decode_phase_tps()))
        cell = {"prompt": pp, "generate": tg,
                "request_gen_tps": round(statistics.median(r[0] for r in runs), 1),
                "prefill_ms": round(statistics.median(r[1] for r in runs), 2),
                "decode_phase_tps": round(statistics.median(r[2] for r in runs), 1)}
        if size == "32b":
            cell["published_request_gen_tps"] = PUBLISHED_32B[(pp, tg)]
            if pp in PUBLISHED_32B_PREFILL_MS:
                cell["published_prefill_ms"] = PUBLISHED_32B_PREFILL_MS[pp]
        cells.append(cell)
    eng.check()
    print(json.dumps({"metric": f"request_gen_tps, one sequence, Qwen3-{size.upper()} layer sizes",
                      "unit": "tok/s", "dtype": "bf16", "data": "synthetic", "reps": reps,
                      "layers": cfg["num_hidden_layers"], "cells": cells}))
    return 0


# Layer sizes for --designs: (width, query heads, kv heads, head size, gated feed-forward rows,
# layers, vocabulary).  The Suvazen model of a size has the same width, heads and layers, a
# feed-forward of 3/2 the rows (two matrices instead of three: the same weights), a rotation of
# half of every head with scaled frequencies, capped scores, sinks, no window (the same keys
# as the Qwen3 model sees), one pass over layers 2-3 with its added vector, capped logits.
DESIGN_SIZES = {"1b": (2048, 16, 8, 128, 6144, 16, 65536),
                "4b": (2560, 32, 8, 128, 9728, 36, 151936),
                "8b": (4096, 32, 8, 128, 12288, 36, 151936)}


def sonalorn_config(size: str) -> dict:
    """The Sonalorn model of a size: the width, heads, head size, layers and vocabulary of
    the Qwen3 model; of every four layers three mix by the gated delta rule (as many heads
    as the attention has, keys and values of the head size, four taps) and one by
    attention; every other layer has a dense feed-forward of the same rows and the rest
    route two of eight experts of a quarter of the rows each (plus one pass-through
    output, three groups of which two are kept): the weights a token uses are below the
    Qwen3 model's, the weights held are above them."""
    W, nq, nkv, D, I, L, V = DESIGN_SIZES[size]
    delta = dict(heads=nq, kv_heads=nkv, dim=D, vdim=D, conv=4)
    attn = dict(heads=nq, kv_heads=nkv, dim=D, vdim=D, scale=D ** -0.5, q_temp={"coef": 0.1, "every": 256})
    dense = {"kind": "dense", "ff": I}
    moe = {"kind": "moe", "expert": {"ff": I // 4 // 64 * 64, "limit": 7.0},
           "router": {"experts": 8, "identity": 1, "top": 2, "groups": {"count": 3, "keep": 2}}}
    layers = [dict(type="attention" if i % 4 == 3 else "delta", mixer=attn if i % 4 == 3 else delta,
                   mlp=dense if i % 2 == 0 else moe) for i in range(L)]
    return dict(architecture="Sonalorn", vocab=V, width=W, max_positions=CONTEXT, norm={"eps": 1e-6},
                layers=layers)


def zutazen_config(size: str) -> dict:
    """The Zutazen model of a size: the width, heads, head size, layers and vocabulary of
    the Qwen3 model; the layers mix in turn by retention (as many heads as the attention
    has, keys and values of the head size, decays from 1 - 2^-5 to 1 - 2^-10), by the
    gated linear recurrence (as many channels as the stream, parts of a head's size, four
    taps) and by latent attention (a latent of 96 and a rotated part of 32, which make a
    cached row of the head size, a window of 1,024); every other layer has a dense
    feed-forward of the same rows and the rest route two of eight experts of a quarter of
    the rows each."""
    W, nq, _nkv, D, I, L, V = DESIGN_SIZES[size]
    ret = dict(heads=nq, dim=D, vdim=D, rot={"base": 1000000.0, "dims": D},
               decay=[1.0 - 2.0 ** (-5.0 - 5.0 * h / max(nq - 1, 1)) for h in range(nq)])
    rec = dict(width=W, blocks=W // D, conv=4)
    lat = dict(heads=nq, dim=D, rot_dim=32, vdim=D, kv_rank=96, scale=(D + 32) ** -0.5,
               rot={"base": 500000.0, "dims": 32}, mask={"size": 1024})
    kinds = (("retention", ret), ("rglru", rec), ("latent_attention", lat))
    dense = {"kind": "dense", "ff": I}
    moe = {"kind": "moe", "expert": {"ff": I // 4 // 64 * 64}, "router": {"experts": 8, "top": 2}}
    layers = [dict(type=kinds[i % 3][0], mixer=kinds[i % 3][1], mlp=dense if i % 2 == 0 else moe)
              for i in range(L)]
    return dict(architecture="Zutazen", vocab=V, width=W, norm={"eps": 1e-6}, embedding={"scale": W ** 0.5},
                layers=layers)


def mananex_config(size: str) -> dict:
    """The Mananex model of a size: the width, heads, head size, layers and vocabulary of
    the Qwen3 model; every layer's mixer is attention (the Qwen3 model's heads, half of
    every head rotated, a window of 1,024 that keeps the first eight tokens, sinks, a gate per
    head) beside forget-gate linear attention (half as many heads, keys of half the head
    size, values of the head size); every other layer has a dense feed-forward of the same
    rows and the rest route two of eight experts of a quarter of the rows each; every
    sublayer's result passes a residual gate of the stream's width, and the stream is the
    depth average of all layers' results."""
    W, nq, nkv, D, I, L, V = DESIGN_SIZES[size]
    left = dict(heads=nq, kv_heads=nkv, dim=D, vdim=D, scale=D ** -0.5, rot={"base": 500000.0, "dims": D // 2},
                mask={"size": 1024, "keep_first": 8})
    right = dict(heads=nq // 2, dim=D // 2, vdim=D)
    mixer = dict(left=left, right=right, left_scale=0.7, right_scale=1.1)
    dense = {"kind": "dense", "ff": I}
    moe = {"kind": "moe", "expert": {"ff": I // 4 // 64 * 64}, "router": {"experts": 8, "top": 2}}
    layers = [dict(type="parallel", mixer=mixer, mlp=dense if i % 2 == 0 else moe) for i in range(L)]
    return dict(architecture="Mananex", vocab=V, width=W, norm={"eps": 1e-6}, layers=layers)


def kakotar_config(size: str) -> dict:
    """The Kakotar model of a size: the width, heads, head size, layers and vocabulary of
    the Qwen3 model; the layers mix in turn by differential attention in chunks of 1,280 (a
    token behind a prompt of 2,048 then sees 768 keys and more; the Qwen3 model's heads, two
    maps of half the head size over values of the head size), by lightning attention (as
    many heads, keys and values of the head size, decays from 1 - 2^-5 to 1 - 2^-10), by
    attention over a window of 1,024 with a YaRN-stretched rotation, and by attention over
    the keys and values of the layer before; every layer routes two of eight experts (four
    groups of which two are kept) beside a shared one, each of 3/8 the Qwen3 model's
    feed-forward rows (two matrices instead of three: the weights of a gated expert of a
    quarter of the rows)."""
    W, nq, nkv, D, I, L, V = DESIGN_SIZES[size]
    ff = 3 * I // 8 // 64 * 64
    diff = dict(heads=nq, kv_heads=nkv, dim=D // 2, vdim=D, scale=(D // 2) ** -0.5, diff=0.5, mask={"size": 1280},
                rot={"base": 500000.0, "dims": D // 2,
                     "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}})
    light = dict(heads=nq, dim=D, vdim=D,
                 decay=[1.0 - 2.0 ** (-5.0 - 5.0 * h / max(nq - 1, 1)) for h in range(nq)])
    attn = dict(heads=nq, kv_heads=nkv, dim=D, vdim=D, scale=D ** -0.5, mask={"size": 1024},
                rot={"base": 1000000.0, "dims": D,
                     "scaling": {"factor": 4.0, "fast": 32.0, "slow": 1.0, "original": 8192}})
    mlp = {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": ff},
           "router": {"experts": 8, "top": 2, "scale": 2.5, "groups": {"count": 4, "keep": 2}}}
    kinds = lambda i: (("attention_2", diff), ("lightning", light), ("attention", attn),
                       ("attention", dict(attn, kv_from=i - 1)))[i % 4]
    layers = [dict(type=kinds(i)[0], mixer=kinds(i)[1], mlp=mlp) for i in range(L)]
    return dict(architecture="Kakotar", vocab=V, width=W, norm={"eps": 1e-6}, layers=layers)


def keralix_config(size: str) -> dict:
    """The Keralix model of a size: the width, heads, head size, layers, feed-forward rows and
    vocabulary of the Qwen3 model, on four residual streams; the layers mix in turn by latent
    attention (a latent of 128 for keys and values, which makes a cached row of the head size, and
    one of 3/8 of the width for the queries, sinks, a gate), by the delta rule with a decay per
    channel (as many heads, keys and values of the head size, four taps, thin products of a
    head's inner size) and by attention behind convolutions of four taps over a window of 1,024
    (the Qwen3 model's heads, every head rotated whole, capped scores, values that are the keys)."""
    W, nq, nkv, D, I, L, V = DESIGN_SIZES[size]
    lat = dict(heads=nq, dim=D, vdim=D, kv_rank=128, q_rank=3 * W // 8 // 64 * 64, scale=D ** -0.5)
    delta = dict(heads=nq, kv_heads=nq, dim=D, vdim=D, conv=4)
    attn = dict(heads=nq, kv_heads=nkv, dim=D, vdim=D, conv=4, scale=D ** -0.5, softcap=50.0,
                mask={"size": 1024}, rot={"base": 1000000.0, "dims": D})
    kinds = (("latent_attention", lat), ("channel_delta", delta), ("attention", attn))
    layers = [dict(type=kinds[i % 3][0], mixer=kinds[i % 3][1], mlp={"kind": "dense", "ff": I}) for i in range(L)]
    return dict(architecture="Keralix", vocab=V, width=W, streams=4, norm={"eps": 1e-6},
                embedding={"scale": W ** 0.5}, layers=layers)


def design_configs(size: str, design: str = "suvazen"):
    W, nq, nkv, D, I, L, V = DESIGN_SIZES[size]
    qwen = dict(QWEN3_4B, hidden_size=W, num_attention_heads=nq, num_key_value_heads=nkv, head_dim=D,
                intermediate_size=I, num_hidden_layers=L, vocab_size=V, tie_word_embeddings=False)
    mixer = dict(heads=nq, kv_heads=nkv, dim=D, vdim=D, scale=D ** -0.5, softcap=30.0,
                 rot={"dims": D // 2, "base": 1000000.0,
                      "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}})
    suv = dict(architecture="Suvazen", vocab=V, width=W, norm={"eps": 1e-6}, residual_mult=0.8,
               logit_scale=0.25, logit_softcap=30.0, loop={"start": 2, "stop": 4, "times": 1},
               layers=[dict(type="attention", mixer=mixer, mlp={"kind": "dense", "ff": 3 * I // 2})
                       for _ in range(L)])
    if design == "sonalorn":
        return {"qwen3": qwen, "sonalorn": sonalorn_config(size)}
    if design == "zutazen":       # beside the attention model and beside the other design with state and experts
        return {"qwen3": qwen, "sonalorn": sonalorn_config(size), "zutazen": zutazen_config(size)}
    if design == "mananex":       # beside the attention model and beside the design with matrix states and experts
        return {"qwen3": qwen, "zutazen": zutazen_config(size), "mananex": mananex_config(size)}
    if design == "kakotar":       # the same two: attention, and matrix states, windows and experts
        return {"qwen3": qwen, "zutazen": zutazen_config(size), "kakotar": kakotar_config(size)}
    if design == "keralix":       # beside attention, beside the other delta rule, beside the other latent attention
        return {"qwen3": qwen, "sonalorn": sonalorn_config(size), "zutazen": zutazen_config(size),
                "keralix": keralix_config(size)}
    return {"qwen3": qwen, "suvazen": suv}


def run_designs(sizes, batch: int, steps: int, warm: int, with_ops: bool, pk,
                which: str = "suvazen", only=None) -> int:
    """Prefill of one 2,048-token prompt and decode steps of ``batch`` sequences that hold such
    prompts, for both designs at each size: device times between CUDA events, the prompt step
    as the median of six after three, the decode steps as generation runs them (tokens chosen
    on the device feed the next captured step).  Weights (GBs) dwarf the L2, nothing is flushed."""
    import torch
    from grout_b200.engine import Engine
    from grout_b200.kernels import ops
    out = {}
    for size in sizes:
        out[size] = {}
        for design, cfg in design_configs(size, which).items():
            if only and design not in only:
                continue
            V = cfg.get("vocab_size", cfg.get("vocab"))
            room = (PROMPT + warm + steps + 64 + 63) // 64 * 64
            eng = Engine.random(cfg, 0, dtype="bfloat16", max_tokens=batch * room, max_batch=batch,
                                max_seq_len=CONTEXT)
            g = torch.Generator().manual_seed(1)

            def prompt():
                return torch.randint(0, V, (PROMPT,), generator=g).tolist()

            times = []
            for i in range(9):
                s = eng.open_sequence()
                torch.cuda.synchronize()
                a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                a.record()
                eng.step([(s, prompt())], [[PROMPT - 1]])
                b.record()
                torch.cuda.synchronize()
                eng.close_sequence(s)
                if i >= 3:
                    times.append(a.elapsed_time(b))
            pre_ms = statistics.median(times)
            slots = [eng.open_sequence() for _ in range(batch)]
            for i in range(0, batch, 8):
                eng.step([(s, prompt()) for s in slots[i:i + 8]])
            first = torch.randint(0, V, (batch,), generator=g).tolist()
            logits = eng.step([(s, [first[j]]) for j, s in enumerate(slots)], [[0]] * batch)
            torch.cuda.synchronize()
            time.sleep(SETTLE_S)
            greedy = [eng.default_sampling()] * batch
            entries = [(s, j) for j, s in enumerate(slots)]
            for i in range(warm):
                logits = eng.step_ahead(entries, eng.choose_ahead(logits, greedy, [0.0] * batch))
            torch.cuda.synchronize()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            for i in range(steps):
                logits = eng.step_ahead(entries, eng.choose_ahead(logits, greedy, [0.0] * batch))
            b.record()
            torch.cuda.synchronize()
            dec_ms = a.elapsed_time(b) / steps
            n_weights = sum(t.numel() for t in _weights_of(eng))
            stores = [x for st in eng.cache.stores for x in getattr(st, "stores", [st])]   # (a layer may have two needs)
            # every layer reads the keys and values its query sees once, those of another layer's
            # cache too; a window or a chunk bounds them, whatever the sequence holds
            layout, ctx_mid = eng.cache.layout, PROMPT + warm + steps / 2
            kv_bytes = 0
            for k, e in enumerate(eng.model.plan.schedule):
                owner = k if e.cache_of is None else e.cache_of
                if owner in layout.where:
                    st = eng.cache.stores[layout.where[owner][0]]
                    kv_bytes += sum(x.k[:1, :1].numel() * 2 * 2 // 64 * _keys_seen(x.spec, ctx_mid)
                                    for x in getattr(st, "stores", [st]) if hasattr(x, "k"))
            # a recurrent mixer reads and writes its whole state every step
            state_bytes = sum(2 * st.state[:, :1].numel() * 4 for st in stores if hasattr(st, "state"))
            step_bytes = 2 * n_weights + batch * (kv_bytes + state_bytes)
            out[size][design] = {
                "prefill_ms": round(pre_ms, 3), "prefill_tok_s": round(PROMPT / pre_ms * 1e3, 1),
                "decode_ms_per_step": round(dec_ms, 4), "decode_tok_s": round(batch / dec_ms * 1e3, 1),
                "weights_gb": round(2 * n_weights / 1e9, 2),
                "decode_hbm_frac": round(step_bytes / (dec_ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
            if with_ops:
                # a fresh engine: its first captured step is the one the timeline traces
                eng.check()
                del eng, logits
                torch.cuda.empty_cache()
                eng = Engine.random(cfg, 0, dtype="bfloat16", max_tokens=batch * room, max_batch=batch,
                                    max_seq_len=CONTEXT)
                logits = None
                slots = [eng.open_sequence() for _ in range(batch)]
                eng.use_graphs = False
                for what in ("prompt step", "decode step"):
                    if what == "decode step":
                        for s in slots:
                            eng.close_sequence(s)
                        slots = [eng.open_sequence() for _ in range(batch)]
                        eng.step([(s, prompt()) for s in slots])
                    run = (lambda: eng.step([(slots[0], prompt())], [[PROMPT - 1]])) if what == "prompt step" \
                        else (lambda: eng.step([(s, [1]) for s in slots], [[0]] * batch))
                    run()
                    if what == "prompt step":
                        eng.close_sequence(slots[0])
                        slots[0] = eng.open_sequence()
                    prof = ops.OpProfile(pk["hbm_gbs"], pk["bf16_tflops"])
                    ops.set_profile(prof)
                    run()
                    ops.set_profile(None)
                    print(f"== {design} at the {size} sizes, {what}" +
                          (f" of {PROMPT} tokens" if what == "prompt step" else
                           f", batch {batch}, {PROMPT} keys a sequence") +
                          f" (peaks: {pk['source']}, {pk['hbm_gbs']:.0f} GB/s, {pk['bf16_tflops']:.0f} TFLOP/s)")
                    print(prof.report())
                print(f"== {design} at the {size} sizes")
                print(decode_timeline(eng, slots, V, g, pk))
            eng.check()
            del eng, logits
            torch.cuda.empty_cache()
    print(json.dumps({"metric": f"prefill and decode throughput, {which.capitalize()} beside Qwen3 at equal layer sizes",
                      "unit": "tok/s", "dtype": "bf16", "data": "synthetic", "batch": batch,
                      "prompt_len": PROMPT, "steps": steps, "warmup": warm, "peaks": pk["source"],
                      "sizes": out}))
    return 0


def _keys_seen(spec, length: float) -> float:
    """The keys that the last token of a sequence of ``length`` sees in this store: all of them, its
    window with the first tokens the window keeps, or those of its chunk so far."""
    if spec.window:
        return min(length, spec.window + spec.keep_first)
    return (length - 1) % spec.chunk + 1 if spec.chunk else length


def _weights_of(eng):
    """Every tensor a step of the engine's model reads as a weight, once."""
    seen, out = set(), []

    def walk(part):
        for v in vars(part).values():
            ts = [v] if hasattr(v, "data_ptr") else ([v.weight] if hasattr(v, "weight") and
                                                     hasattr(getattr(v, "weight"), "data_ptr") else [])
            for t in ts:
                if t.data_ptr() not in seen:
                    seen.add(t.data_ptr())
                    out.append(t)
        for c in part.children():
            walk(c)

    for top in [eng.model.embedding, *eng.model.blocks, eng.model.final_norm, eng.model.head]:
        walk(top)
    emb = eng.model.embedding.weight
    return [t for t in out if t.data_ptr() != emb.data_ptr() or getattr(eng.model.head, "tied", False)]


def quartiles(xs):
    xs = sorted(xs)
    q = statistics.quantiles(xs, n=4, method="inclusive") if len(xs) > 1 else [xs[0]] * 3
    return q[0], q[1], q[2]


def run_ops(size: str, batch: int, layers: int, pk) -> int:
    """One prompt step of 2,048 tokens launched kernel by kernel with an event pair
    around each (the table of ``ops.OpProfile``: every kernel alone on the device),
    and the decode step of ``batch`` sequences as it runs inside its captured graph
    (``decode_timeline``)."""
    import torch
    from grout_b200.engine import Engine
    from grout_b200.kernels import ops
    cfg = dict(SIZES[size], num_hidden_layers=layers)
    eng = Engine.random(cfg, 0, dtype="bfloat16", max_tokens=batch * (PROMPT + 128),
                        max_batch=batch, max_seq_len=CONTEXT)
    eng.use_graphs = False
    g = torch.Generator().manual_seed(1)
    V = cfg["vocab_size"]

    def prompt():
        return torch.randint(0, V, (PROMPT,), generator=g).tolist()

    slots = [eng.open_sequence() for _ in range(batch)]
    eng.step([(slots[0], prompt())], [[PROMPT - 1]])                  # warm-up of every prompt kernel
    eng.close_sequence(slots[0])
    slots[0] = eng.open_sequence()
    prof = ops.OpProfile(pk["hbm_gbs"], pk["bf16_tflops"])
    ops.set_profile(prof)
    eng.step([(slots[0], prompt())], [[PROMPT - 1]])
    ops.set_profile(None)
    print(f"== prompt step, {PROMPT} tokens, Qwen3-{size.upper()} layer sizes, {layers} layers "
          f"(peaks: {pk['source']}, {pk['hbm_gbs']:.0f} GB/s, {pk['bf16_tflops']:.0f} TFLOP/s burst)")
    print(prof.report())
    for i in range(1, batch, 8):
        eng.step([(s, prompt()) for s in slots[i:i + 8]])
    eng.check()
    print(decode_timeline(eng, slots, V, g, pk))
    return 0


def decode_timeline(eng, slots, V, g, pk, steps: int = 3) -> str:
    """The kernels of a captured decode step as they ran inside it, from the activity
    records of the CUDA profiling interface (torch.profiler): per kernel its calls a
    step, its mean duration, and its mean *exposed* time, which is how much later it
    ended than everything before it (kernels overlap at their edges: a kernel is
    resident, fetching what no earlier kernel writes, while its predecessor drains).
    The exposed times add up to the step.  Times taken under the profiler's tracing:
    a breakdown, not a benchmark figure."""
    import torch
    from torch.profiler import ProfilerActivity, profile
    from grout_b200.kernels import ops
    batch = len(slots)
    eng.use_graphs = True
    tok = torch.randint(0, V, (batch,), generator=g).tolist()

    def step():
        eng.step([(s, [t]) for s, t in zip(slots, tok)], [[0]] * batch)

    # the capture of the step's graph (a warm-up pass and the captured pass) says, launch by
    # launch, which product each kernel of the step is; kernel names alone do not
    eng.graphs.decode_graphs.clear()
    ops.LAUNCH_LOG = []
    step()
    graph = eng.graphs.decode(batch, max(eng.cache.length[s] for s in slots))
    labels = ops.LAUNCH_LOG[-graph.kernels_per_replay:]         # the captured pass
    ops.LAUNCH_LOG = None
    for _ in range(5):
        step()
    torch.cuda.synchronize()
    with profile(activities=[ProfilerActivity.CUDA]) as prof:
        for _ in range(steps):
            step()
        torch.cuda.synchronize()
    ev = sorted((e for e in prof.events() if e.device_type == torch.autograd.DeviceType.CUDA
                 and "memcpy" not in e.name.lower() and "memset" not in e.name.lower()),
                key=lambda e: e.time_range.start)
    # a step begins with its embedding kernel, whichever the model has
    starts = [i for i, e in enumerate(ev) if any(k in e.name for k in ("embed_kernel", "embed_pos_norm_kernel", "embed_scaled_kernel"))]
    rows, total = {}, 0.0
    for a, b in zip(starts, starts[1:] + [len(ev)]):
        frontier = ev[a].time_range.start
        named = len(labels) == b - a
        for k, e in enumerate(ev[a:b]):
            end = e.time_range.end
            name = labels[k] if named else e.name.split("(")[0].replace("void ", "")
            r = rows.setdefault(name, [0, 0.0, 0.0])
            r[0] += 1
            r[1] += end - e.time_range.start
            r[2] += max(0.0, end - frontier)
            frontier = max(frontier, end)
        total += frontier - ev[a].time_range.start
    n = len(starts)
    if n and len(labels) != len(ev) // n:
        print(f"bench.py: {len(labels)} launches were logged for a step of {len(ev) // n} kernels; "
              f"rows are named by kernel", file=sys.stderr)
    kv_spec = next((x.spec for st in eng.cache.stores for x in getattr(st, "stores", [st]) if hasattr(x, "k")), None)
    kv = sum(int(_keys_seen(kv_spec, eng.cache.length[s])) if kv_spec is not None else 0 for s in slots)

    def must_read(name):
        """Bytes a call of this kernel has to read: a product its weights, the decode
        attention the keys and values of the live sequences (one layer's)."""
        part = name.split()
        if part[0] == "gemm_tc_bf16" and len(part) > 1 and "x" in part[1]:
            rows_w, cols_w = part[1].split("x")
            return 2.0 * int(rows_w) * int(cols_w)
        if part[0].startswith("attn_decode") and "second" not in name:
            return 2.0 * kv * 2 * kv_spec.n_kv_heads * kv_spec.head_dim
        return None

    lines = [f"== decode step, batch {batch}, {kv // batch} keys a sequence in reach, as it ran inside the captured "
             f"graph ({n} steps traced): {total / n:.1f} us a step; GB/s = what the kernel has to read / "
             f"its exposed time, of the {pk['source']} {pk['hbm_gbs']:.0f} GB/s",
             f"  {'kernel':<36}{'calls/step':>11}{'mean_us':>9}{'exposed_us':>11}{'per step':>10}{'share':>7}"
             f"{'GB/s':>8}{'of hbm':>8}"]
    for name, (calls, dur, exposed) in sorted(rows.items(), key=lambda kv: -kv[1][2]):
        line = (f"  {name[:35]:<36}{calls / n:>11.1f}{dur / calls:>9.2f}{exposed / calls:>11.2f}"
                f"{exposed / n:>10.1f}{exposed / total:>7.1%}")
        nbytes = must_read(name)
        if nbytes and exposed > 0:
            gbs = nbytes / (exposed / calls * 1e-6) / 1e9
            line += f"{gbs:>8.0f}{gbs / pk['hbm_gbs']:>8.2f}"
        lines.append(line)
    return "\n".join(lines)


def main() -> int:
    global PROMPT, CONTEXT
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=128)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--size", default="4b", choices=sorted(SIZES),
                    help="layer sizes of the run (default: the 4B sizes the contract names)")
    ap.add_argument("--layers", type=int, default=None,
                    help="fewer layers than the configuration has (both numbers are reported)")
    ap.add_argument("--prompt-len", type=int, default=PROMPT,
                    help="tokens every sequence holds before decoding, and of the timed prompt step "
                         "(default: the 2,048 the contract names; other lengths for the profiles)")
    ap.add_argument("--no-points", action="store_true", help="skip decode at batch 1 and 64")
    ap.add_argument("--phases", default="prefill,decode,points,e2e",
                    help="which measurements to run (a profiler wants one at a time)")
    ap.add_argument("--requests", default=None, choices=sorted(SIZES),
                    help="instead of the default run: the reference's request grid at this model size")
    ap.add_argument("--reps", type=int, default=5, help="measured requests per cell of --requests")
    ap.add_argument("--ops", action="store_true",
                    help="instead of the default run: the per-kernel table of a prompt step and of "
                         "decode steps at --size and --batch")
    ap.add_argument("--designs", action="store_true",
                    help="instead of the default run: the Suvazen design beside the Qwen3 decoder at "
                         "equal layer sizes (--design-sizes), prefill and decode at --batch")
    ap.add_argument("--design", default="suvazen", choices=["suvazen", "sonalorn", "zutazen", "mananex", "kakotar", "keralix"],
                    help="which design --designs sets beside Qwen3")
    ap.add_argument("--design-sizes", default="1b,4b,8b",
                    help=f"which of {sorted(DESIGN_SIZES)} --designs runs")
    ap.add_argument("--design-models", default=None,
                    help="with --designs: run only these of the models it would run (comma-separated names)")
    ap.add_argument("--design-ops", action="store_true",
                    help="with --designs: also the per-kernel tables of a prompt step and a decode step")
    args = ap.parse_args()

    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "NikVisel/grout is a Rust crate (Cargo.toml, no Python packaging); pip "
                          "cannot install it offline and no Rust toolchain or crates are present"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py: this library runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    if args.requests:
        return run_requests(args.requests, max(1, args.reps))
    if args.designs:
        sizes = [x for x in args.design_sizes.split(",") if x]
        if any(x not in DESIGN_SIZES for x in sizes):
            print(f"bench.py: --design-sizes takes {sorted(DESIGN_SIZES)}", file=sys.stderr)
            return 2
        only = [x for x in args.design_models.split(",") if x] if args.design_models else None
        return run_designs(sizes, args.batch, min(args.steps, 64), max(args.warmup, 3), args.design_ops,
                           peaks(), args.design, only)
    if args.prompt_len != PROMPT:
        if not 1 <= args.prompt_len <= 36864:
            print("bench.py: --prompt-len must be 1..36864", file=sys.stderr)
            return 2
        PROMPT = args.prompt_len
        CONTEXT = max(CONTEXT, (PROMPT + 2048 + 63) // 64 * 64)
    full_layers = SIZES[args.size]["num_hidden_layers"]
    layers = args.layers or full_layers
    pk = peaks()
    if args.ops:
        return run_ops(args.size, args.batch, layers, pk)
    W = max(args.warmup, 3)
    K = args.steps
    most = CONTEXT - PROMPT - W - 4      # the sequences hold 2,048 prompt tokens in a context of 4,096
    if K < 1 or K > most:
        print(f"bench.py: --steps must be 1..{most} with --warmup {W} (prompt {PROMPT}, context "
              f"{CONTEXT}); got {K}", file=sys.stderr)
        return 2
    phases = set(args.phases.split(","))
    if args.no_points:
        phases.discard("points")

    import torch
    from grout_b200.engine import Engine
    from grout_b200.kernels import ops

    cfg = dict(SIZES[args.size], num_hidden_layers=layers)
    torch.manual_seed(0)
    room = PROMPT + max(W + K, 129) + 64
    point_batches = [1, 64] if "points" in phases else []
    # (a cache for 64 sequences of a long prompt does not fit beside the weights: such a
    # run keeps the batch-1 point only)
    if 64 * room * kv_bytes_per_token(cfg, layers) > 100e9:
        point_batches = [b for b in point_batches if b * room * kv_bytes_per_token(cfg, layers) <= 100e9]
    biggest = max([args.batch] + point_batches)
    eng = Engine.random(cfg, 0, dtype="bfloat16", max_tokens=biggest * ((room + 63) // 64 * 64),
                        max_batch=biggest, max_seq_len=CONTEXT)
    g = torch.Generator().manual_seed(1)
    V = cfg["vocab_size"]

    def prompt():
        return torch.randint(0, V, (PROMPT,), generator=g).tolist()

    def ev():
        return torch.cuda.Event(enable_timing=True)

    # ---- prefill of 2,048 tokens ---------------------------------------------------
    p = prompt()
    times = []
    for i in range(9 if "prefill" in phases else 0):      # three to warm up, the median of six
        s = eng.open_sequence()
        torch.cuda.synchronize()
        a, b = ev(), ev()
        a.record()
        eng.step([(s, p)], [[PROMPT - 1]])
        b.record()
        torch.cuda.synchronize()
        eng.close_sequence(s)
        if i >= 3:
            times.append(a.elapsed_time(b))
    prefill = None
    if times:
        pre_ms = statistics.median(times)
        rate = prefill_flops(cfg, layers, PROMPT) / (pre_ms * 1e-3) / 1e12
        # the step's flops / time / the peak of its dtype: against the burst peak (a product
        # timed alone) and against the sustained one (nine prompt steps back to back run at
        # the clocks of the power cap, as that peak was taken)
        prefill = {"value": round(PROMPT / pre_ms * 1e3, 1), "tokens": PROMPT, "ms": round(pre_ms, 3),
                   "frac": round(rate / pk["bf16_tflops"], 4),
                   "frac_sustained": round(rate / pk["bf16_tflops_sustained"], 4),
                   "tflops": round(rate, 1), "of": pk["source"]}

    # ---- decode --------------------------------------------------------------------
    def decode_run(batch, steps, warm, sample_clocks=False):
        slots = [eng.open_sequence() for _ in range(batch)]
        group = max(1, min(8, 16384 // PROMPT))            # prompts go in, 16,384 tokens at a time
        for i in range(0, batch, group):
            eng.step([(s, prompt()) for s in slots[i:i + group]])
        # the decode step as generation runs it: tokens chosen on the device (greedy)
        # feed the next step, which is queued without waiting for the host
        first = torch.randint(0, V, (batch,), generator=g).tolist()
        logits = eng.step([(s, [first[j]]) for j, s in enumerate(slots)], [[0]] * batch)
        # The prompts leave the GPU at the reduced clocks of its power cap, and it raises
        # them again over some thirty decode steps; the decode step is measured at the
        # clocks it settles at, so the GPU idles for half a second first.  (``e2e`` below
        # has no such pause: it is the request as a user runs it.)
        torch.cuda.synchronize()
        time.sleep(SETTLE_S)
        greedy = [eng.default_sampling()] * batch
        entries = [(s, j) for j, s in enumerate(slots)]
        for i in range(warm):
            logits = eng.step_ahead(entries, eng.choose_ahead(logits, greedy, [0.0] * batch))
        torch.cuda.synchronize()
        clocks = ClockSampler() if sample_clocks else None
        if clocks:
            clocks.start()
        before = ops.launch_count()
        cuts = sorted({round(steps * r / REGIONS) for r in range(1, REGIONS)} - {0, steps})
        marks = [ev()]
        marks[0].record()
        for i in range(steps):
            logits = eng.step_ahead(entries, eng.choose_ahead(logits, greedy, [0.0] * batch))
            if i + 1 in cuts:
                marks.append(ev())
                marks[-1].record()
        marks.append(ev())
        marks[-1].record()
        torch.cuda.synchronize()
        ms = marks[0].elapsed_time(marks[-1])
        bounds = [0] + cuts + [steps]
        per_step = [a.elapsed_time(b) / (hi - lo)
                    for a, b, lo, hi in zip(marks, marks[1:], bounds, bounds[1:])]
        launches = ops.launch_count() - before
        graph = eng.graphs.decode(batch, PROMPT + warm + steps + 1)
        if graph is not None and graph.graph is not None:
            launches += steps * graph.kernels_per_replay
        ctx_mid = PROMPT + warm + steps / 2.0
        for s in slots:
            eng.close_sequence(s)
        return ms, launches, ctx_mid, (clocks.stop() if clocks else None), per_step

    def step_bytes(batch, ctx):
        return weight_bytes(cfg, layers) + batch * ctx * kv_bytes_per_token(cfg, layers)

    ms, launches, ctx_mid, clocks, per_step = decode_run(args.batch, K, W, sample_clocks=True)
    value = args.batch * K / ms * 1e3
    achieved = step_bytes(args.batch, ctx_mid) / (ms / K * 1e-3) / 1e9
    roofline = {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"],
                "unit": "GB/s", "frac": round(achieved / pk["hbm_gbs"], 4), "of": pk["source"]}
    q1, med, q3 = quartiles(per_step)
    regions = {"n": len(per_step), "ms_per_step_median": round(med, 4),
               "ms_per_step_q1": round(q1, 4), "ms_per_step_q3": round(q3, 4),
               "value_at_median": round(args.batch / med * 1e3, 1)}

    points = {}
    if point_batches:
        for bsz in point_batches:
            m, _l, c, _, _p = decode_run(bsz, 32, 4)
            points[f"decode_b{bsz}"] = round(bsz * 32 / m * 1e3, 1)
            points[f"decode_b{bsz}_hbm_frac"] = round(
                step_bytes(bsz, c) / (m / 32 * 1e-3) / 1e9 / pk["hbm_gbs"], 4)

    # ---- end to end through the Python entry point -----------------------------------
    e2e = None
    if "e2e" in phases:
        # at least 128 decode steps: the first thirty after the prompts run at the clocks the
        # power cap left behind, and a request of a few tokens would measure little else
        n_new = max(K, 128) + 1
        prompts = [prompt() for _ in range(args.batch)]
        eng.generate(prompts, 4, ignore_eos=True)              # warm-up
        outs = eng.generate(prompts, n_new, ignore_eos=True)
        e2e_tps = sum(o.generated_tokens - 1 for o in outs) / outs[0].decode_elapsed
        graph = eng.graphs.decode(args.batch, PROMPT + n_new)
        h2d = int(graph.dev.numel() * 4) if graph is not None else 0
        e2e = {"value": round(e2e_tps, 1), "unit": "tok/s", "steps": n_new - 1, "h2d_bytes_per_step": h2d,
               "d2h_bytes_per_step": 4 * args.batch}

    eng.check()      # a kernel that gave up on a bounded wait would have voided the numbers
    name = f"Qwen3-{args.size.upper()}"
    print(json.dumps({
        "metric": f"decode tok/s ({name} shape, batch {args.batch}, 2,048-token prompts)",
        "value": round(value, 1), "unit": "tok/s", "n_gpus": 1, "steps": K, "warmup": W,
        "ms_per_step": round(ms / K, 4), "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic", "impl": "ours",
        "config": {"model": f"{name} layer sizes, random weights", "layers": layers,
                   "layers_of_config": full_layers, "hidden": cfg["hidden_size"],
                   "heads": cfg["num_attention_heads"], "kv_heads": cfg["num_key_value_heads"],
                   "head_dim": cfg["head_dim"], "intermediate": cfg["intermediate_size"],
                   "vocab": V, "global_batch": args.batch, "seq_len": CONTEXT,
                   "prompt_len": PROMPT, "tied_head": bool(cfg["tie_word_embeddings"]),
                   "parallelism": "single GPU",
                   "l2": f"inputs larger than L2 ({weight_bytes(cfg, layers) / 1e9:.0f} GB of weights "
                         f"per step), no flush",
                   "settle_s": SETTLE_S, "peaks": pk["source"]},
        "clocks": clocks, "e2e": e2e, "gpu_launches": launches, "prefill": prefill,
        "roofline": roofline, "regions": regions, "points": points}))
    return 0


if __name__ == "__main__":
    sys.exit(main())
