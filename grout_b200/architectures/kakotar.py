"""The Kakotar decoder as a plan.

Pre-norm layers, x <- x + M(N1(x)); x <- x + F(N2(x)), whose norms are dynamic tanhs
(no statistics of a row).  A layer's mixer M is lightning attention (a fading matrix-valued
state per head, activated queries, keys and values, one gated norm over all heads), softmax
attention over a window with a YaRN-stretched rotation, which may read the keys and values
of an earlier such layer, or differential attention within fixed chunks of the sequence
with a rotation stretched band by band.  F is a mixture of small ungated squared-relu
experts with a shared one: sigmoid scores, a correction for the choice, a choice within the
best groups (by their two largest), weights normalised to a constant.  This file holds the
checkpoint's tensor names, the constants the design fixes and the order of the parts; every
size and every other constant comes from the configuration.

Tensor names: ``embed``, ``head``, ``final.norm`` and per layer i ``l<i>.norm1`` / ``norm2``,
each norm with ``.alpha`` and ``.b``; a lightning mixer's ``l<i>.mix.{q,k,v,g,norm,o}``; an
attention mixer's ``l<i>.mix.{q,k,v,o}`` (without k and v where it reads another layer's),
a differential one's also ``lq1``, ``lk1``, ``lq2``, ``lk2``; ``l<i>.mlp.e<j>.{up,down}``,
``router``, ``correction`` and ``shared.{up,down}``.
"""
from __future__ import annotations

from ..config import KakotarConfig, register_architecture
from ..parts.base import PartSpec
from ..parts.plan import LayerPlan, ModelPlan, ScheduleEntry

NO_POSITION_LIMIT = 1 << 30       # nothing in the design bounds a sequence's length


def _norm(dim: int) -> PartSpec:
    return PartSpec("dynamic_tanh", dict(dim=dim, name=""))


def _position(m: dict) -> PartSpec:
    rot = m.get("rot")
    if not rot or not rot["dims"]:
        return PartSpec("none", {})
    return PartSpec("rotary_half_split", dict(
        head_dim=m["dim"], theta=float(rot["base"]), rot_dim=int(rot["dims"]),
        scaling=rot.get("scaling"), exact_table=True))


def _size(m: dict):
    return int(m["mask"]["size"]) if m.get("mask") else None


def _reach(cfg: KakotarConfig, i: int):
    """How many keys back the layers look that read layer i's keys (None: all)."""
    readers = [layer["mixer"] for layer in cfg.layers
               if layer["type"] == "attention" and layer["mixer"].get("kv_from") == i]
    sizes = [_size(m) for m in readers]
    return None if None in sizes else max(sizes, default=0)


def _mixer(cfg: KakotarConfig, i: int) -> PartSpec:
    layer, width, eps = cfg.layers[i], cfg.width, float(cfg.norm["eps"])
    m = layer["mixer"]
    if layer["type"] == "lightning":
        return PartSpec("lightning_attention", dict(
            hidden=width, n_heads=m["heads"], key_dim=m["dim"], value_dim=m["vdim"],
            decay=tuple(float(d) for d in m["decay"]), norm_eps=eps))
    if layer["type"] == "attention_2":
        return PartSpec("differential_attention", dict(
            hidden=width, n_heads=m["heads"], n_kv_heads=m["kv_heads"], head_dim=m["dim"],
            v_head_dim=m["vdim"], position=_position(m), scale=float(m["scale"]),
            diff=float(m["diff"]), norm_eps=eps, chunk=_size(m)))
    return PartSpec("gqa_attention", dict(
        hidden=width, n_heads=m["heads"], n_kv_heads=m["kv_heads"], head_dim=m["dim"],
        v_head_dim=m["vdim"], position=_position(m), scale=float(m["scale"]), window=_size(m),
        shares_kv=m.get("kv_from") is not None, reach=_reach(cfg, i),
        names={"q": "q", "k": "k", "v": "v", "o": "o"}))


def _feedforward(width: int, mlp: dict) -> PartSpec:
    r, g, shared = mlp["router"], mlp["router"].get("groups"), mlp.get("shared")
    return PartSpec("routed_experts", dict(
        hidden=width, intermediate=int(mlp["expert"]["ff"]), n_experts=int(r["experts"]), top=int(r["top"]),
        score_fn="sigmoid", gated=False, n_groups=int(g["count"]) if g else 1,
        keep_groups=int(g["keep"]) if g else 1, group_score="top2", normalize=True,
        weight_scale=float(r["scale"]), shared_intermediate=int(shared["ff"]) if shared else None))


def kakotar_plan(cfg: KakotarConfig) -> ModelPlan:
    W = cfg.width
    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        args = dict(norm1=_norm(W), mixer=_mixer(cfg, i))
        if layer.get("mlp") is not None:
            args.update(norm2=_norm(W), feedforward=_feedforward(W, layer["mlp"]))
        layers.append(LayerPlan(PartSpec("prenorm", args), f"l{i}.", {
            "norm1": "norm1", "norm2": "norm2", "mixer": "mix.", "feedforward": "mlp."}))
        src = layer["mixer"].get("kv_from")
        schedule.append(ScheduleEntry(i, cache_of=None if src is None else int(src)))
    return ModelPlan(
        embedding=PartSpec("token", dict(vocab=cfg.vocab, hidden=W, name="embed", scale=1.0)),
        embedding_prefix="",
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=_norm(W),
        final_norm_prefix="final.norm",
        head=PartSpec("linear", dict(vocab=cfg.vocab, hidden=W, tied=False, name="head")),
        head_prefix="",
        vocab_size=cfg.vocab,
        max_position=NO_POSITION_LIMIT,
        stop_tokens=cfg.eos_token_ids(),
    )


register_architecture("Kakotar", KakotarConfig, kakotar_plan, model_types=("kakotar",))
