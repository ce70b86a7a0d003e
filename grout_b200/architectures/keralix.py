"""The Keralix decoder as a plan.

Pre-norm layers on several residual streams ("hyper-connections"): a sublayer reads a
weighted sum of the streams behind an RMS norm, the streams are mixed with one another, and
the sublayer's result goes back into each of them with a weight of its own; the last norm
reads their sum.  A layer's mixer is windowed attention with short convolutions behind its
query and key projections and values that are the convolved keys, attention without
positions whose queries and keys both come from latent vectors (with a sink and an
elementwise gate), or a delta rule whose state fades by one factor per key channel.  The
feed-forward, where a layer has one, is silu-gated.  The head is the embedding table.  This
file holds the checkpoint's tensor names, the constants the design fixes and the order of
the parts; every size and every other constant comes from the configuration.

Tensor names: ``embed``, ``final.norm`` and per layer i ``l<i>.norm1`` / ``norm2``,
``l<i>.hc1.{in,out,mix}`` / ``hc2``; an attention's ``l<i>.mix.{q,k}`` each with ``.b`` and
``.conv``, ``o``; a latent attention's ``l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,sink,g,o}``;
a delta rule's ``l<i>.mix.{q,k,v}`` each with ``.conv``,
``{b,A_log,a1,a2,dt_bias,g1,g2,norm,o}``; ``l<i>.mlp.{gate,up,down}``.
"""
from __future__ import annotations

from ..config import KeralixConfig, register_architecture
from ..parts.base import PartSpec
from ..parts.plan import LayerPlan, ModelPlan, ScheduleEntry

UNIT_EPS = 1e-6                   # under the root that makes the delta rule's q and k unit vectors
NO_POSITION_LIMIT = 1 << 30       # nothing in the design bounds a sequence's length


def _rms(dim: int, eps: float) -> PartSpec:
    return PartSpec("rmsnorm", dict(dim=dim, eps=eps, name=""))


def _attention(width: int, m: dict) -> PartSpec:
    rot, mask = m.get("rot"), m.get("mask")
    position = (PartSpec("rotary_half_split", dict(head_dim=m["dim"], theta=float(rot["base"]),
                                                   rot_dim=int(rot["dims"]), exact_table=True))
                if rot and rot["dims"] else PartSpec("none", {}))
    return PartSpec("gqa_attention", dict(
        hidden=width, n_heads=m["heads"], n_kv_heads=m["kv_heads"], head_dim=m["dim"],
        position=position, scale=float(m["scale"]), window=int(mask["size"]) if mask else None,
        softcap=m.get("softcap"), values_are_keys=True, qk_bias=True, conv_taps=int(m["conv"]),
        names={"q": "q", "k": "k", "o": "o", "q_bias": "q.b", "k_bias": "k.b", "q_conv": "q.conv",
               "k_conv": "k.conv"}))


def _mixer(kind: str, width: int, m: dict, eps: float) -> PartSpec:
    if kind == "attention":
        return _attention(width, m)
    if kind == "latent_attention":
        return PartSpec("latent_attention", dict(
            hidden=width, n_heads=m["heads"], head_dim=m["dim"], rot_dim=0, v_head_dim=m["vdim"],
            kv_rank=m["kv_rank"], q_rank=m["q_rank"], position=PartSpec("none", {}),
            scale=float(m["scale"]), norm_eps=eps, sinks=True, gated=True))
    return PartSpec("channel_delta", dict(
        hidden=width, n_heads=m["heads"], n_kv_heads=m["kv_heads"], key_dim=m["dim"],
        value_dim=m["vdim"], conv_taps=m["conv"], norm_eps=eps, unit_eps=UNIT_EPS))


def keralix_plan(cfg: KeralixConfig) -> ModelPlan:
    W, eps = cfg.width, float(cfg.norm["eps"])
    layers = []
    for i, layer in enumerate(cfg.layers):
        args = dict(streams=cfg.streams, norm1=_rms(W, eps),
                    mixer=_mixer(layer["type"], W, layer["mixer"], eps), hyper1="hc1.", hyper2="hc2.")
        if layer.get("mlp") is not None:
            args.update(norm2=_rms(W, eps), feedforward=PartSpec("gated_mlp", dict(
                hidden=W, intermediate=int(layer["mlp"]["ff"]), activation="silu", bias=False,
                names={"gate": "gate", "up": "up", "down": "down"})))
        layers.append(LayerPlan(PartSpec("hyper_prenorm", args), f"l{i}.", {
            "norm1": "norm1", "norm2": "norm2", "mixer": "mix.", "feedforward": "mlp."}))
    return ModelPlan(
        embedding=PartSpec("token", dict(vocab=cfg.vocab, hidden=W, name="embed",
                                         scale=float(cfg.embedding["scale"]))),
        embedding_prefix="",
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i) for i in range(len(cfg.layers))),
        final_norm=_rms(W, eps),
        final_norm_prefix="final.norm",
        head=PartSpec("linear", dict(vocab=cfg.vocab, hidden=W, tied=True)),
        head_prefix="",
        vocab_size=cfg.vocab,
        max_position=NO_POSITION_LIMIT,
        stop_tokens=cfg.eos_token_ids(),
    )


register_architecture("Keralix", KeralixConfig, keralix_plan, model_types=("keralix",))
