"""Configuration of the Kakotar decoder.

The file names the design under ``architecture`` and describes the model layer by
layer: ``layers`` is a list of objects ``{"type", "mixer", "mlp"}`` (``mlp`` null or
absent: the layer has no feed-forward).  Nothing that the arithmetic needs is defaulted; a
term whose key is absent (``rot``, ``rot.scaling``, ``mask``, ``router.groups``, ``shared``)
is absent from the model.

    vocab, width                    sizes of the two token tables and of the stream
    norm.eps                        epsilon under the roots (the layers' norms have none)
    layers[i].type                  "lightning" | "attention" | "attention_2"
    layers[i].mixer  (lightning)    heads, dim, vdim, decay (one per head)
    layers[i].mixer  (attention)    heads, kv_heads, dim, vdim, scale, rot.{base, dims, scaling},
                                    mask.size (a window), kv_from (the layer whose keys and
                                    values this one reads)
    layers[i].mixer  (attention_2)  heads, kv_heads, dim, vdim, scale, diff,
                                    rot.{base, dims, scaling}, mask.size (a chunk)
    rot.scaling                     {"factor", "original", "fast", "slow"} or
                                    {"factor", "original", "low", "high"}
    layers[i].mlp                   {"kind": "moe", "expert": {"ff"}, "shared": {"ff"},
                                    "router": {"experts", "top", "scale",
                                    "groups": {"count", "keep"}}}
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .base import ModelConfig

_LAYER_TYPES = ("lightning", "attention", "attention_2")
_MLP_KINDS = ("moe",)
_SCALINGS = (("factor", "original", "fast", "slow"), ("factor", "original", "low", "high"))


def _number(v) -> bool:
    return isinstance(v, (int, float)) and not isinstance(v, bool)


def _positive(v) -> bool:
    return _number(v) and v > 0


def _positive_int(v) -> bool:
    return isinstance(v, int) and not isinstance(v, bool) and v > 0


def _count(v) -> bool:
    return isinstance(v, int) and not isinstance(v, bool) and v >= 0


@dataclass(frozen=True)
class KakotarConfig(ModelConfig):
    vocab: int
    width: int
    layers: Tuple[dict, ...]
    norm: dict
    architecture: str = "Kakotar"
    eos_token_id: Optional[int] = None

    def validate(self):
        for key in ("vocab", "width"):
            if not _positive_int(getattr(self, key)):
                yield f"'{key}' must be a positive integer, found {getattr(self, key)!r}"
        if not _positive(self.norm.get("eps")):
            yield f"'norm.eps' must be a positive number, found {self.norm.get('eps')!r}"
        if not self.layers:
            yield "'layers' is empty"
        for i, layer in enumerate(self.layers):
            yield from self._layer_problems(i, layer)

    def _layer_problems(self, i, layer):
        where = f"layers[{i}]"
        if not isinstance(layer, dict):
            yield f"{where} is not an object"
            return
        if layer.get("type") not in _LAYER_TYPES:
            yield f"{where}.type={layer.get('type')!r}: this design has {list(_LAYER_TYPES)}"
            return
        m = layer.get("mixer")
        if not isinstance(m, dict):
            yield f"{where}.mixer is missing"
            return
        sizes = ("heads", "dim", "vdim") if layer["type"] == "lightning" else ("heads", "kv_heads", "dim", "vdim")
        bad = [k for k in sizes if not _positive_int(m.get(k))]
        for key in bad:
            yield f"{where}.mixer.{key} must be a positive integer, found {m.get(key)!r}"
        if not bad:
            if layer["type"] == "lightning":
                yield from self._lightning_problems(where + ".mixer", m)
            else:
                yield from self._attention_problems(i, where + ".mixer", layer["type"], m)
        yield from self._mlp_problems(where, layer.get("mlp"))

    def _lightning_problems(self, where, m):
        decay = m.get("decay")
        if not isinstance(decay, (list, tuple)) or len(decay) != m["heads"] or not all(_number(d) for d in decay):
            yield f"{where}.decay needs a number for each of {m['heads']} heads, found {decay!r}"

    def _attention_problems(self, i, where, kind, m):
        if m["heads"] % m["kv_heads"]:
            yield f"{where}: {m['heads']} heads cannot share {m['kv_heads']} kv heads"
        for key in ("scale", "diff") if kind == "attention_2" else ("scale",):
            if not _number(m.get(key)):
                yield f"{where}.{key} must be a number, found {m.get(key)!r}"
        rot = m.get("rot")
        if rot is not None:
            if not (isinstance(rot, dict) and _positive(rot.get("base"))
                    and _count(rot.get("dims")) and rot["dims"] % 2 == 0):
                yield f"{where}.rot needs a positive 'base' and an even 'dims', found {rot!r}"
            else:
                if rot["dims"] > m["dim"]:
                    yield f"{where}.rot.dims={rot['dims']} exceeds the head's {m['dim']} elements"
                s = rot.get("scaling")
                if s is not None and not (isinstance(s, dict) and
                                          any(all(_positive(s.get(k)) for k in keys) for keys in _SCALINGS)):
                    yield f"{where}.rot.scaling needs positive numbers {' or '.join(map(str, _SCALINGS))}, found {s!r}"
        mask = m.get("mask")
        if mask is not None and not (isinstance(mask, dict) and _positive_int(mask.get("size"))):
            yield f"{where}.mask needs a positive integer 'size', found {mask!r}"
        src = m.get("kv_from")
        if src is None:
            return
        if kind != "attention":
            yield f"{where}.kv_from: only layers of type 'attention' read another layer's keys and values"
            return
        if not _count(src) or src >= i:
            yield f"{where}.kv_from={src!r} must name an earlier layer"
            return
        other = self.layers[src]
        om = other.get("mixer") if isinstance(other, dict) else None
        if not isinstance(om, dict) or other.get("type") != "attention" or om.get("kv_from") is not None:
            yield f"{where}.kv_from={src} must name a layer of type 'attention' with projections of its own"
            return
        for key in ("kv_heads", "dim", "vdim"):
            if om.get(key) != m[key]:
                yield f"{where}.{key}={m[key]} differs from the {om.get(key)!r} of layer {src}, whose keys it reads"

    def _mlp_problems(self, where, mlp):
        if mlp is None:
            return
        if not isinstance(mlp, dict) or mlp.get("kind") not in _MLP_KINDS:
            yield f"{where}.mlp.kind={mlp!r}: this design has {list(_MLP_KINDS)}"
            return
        for key in ("expert", "shared"):
            part = mlp.get(key)
            if part is None and key == "shared":
                continue
            if not (isinstance(part, dict) and _positive_int(part.get("ff"))):
                yield f"{where}.mlp.{key} needs a positive integer 'ff', found {part!r}"
        r = mlp.get("router")
        if not (isinstance(r, dict) and _positive_int(r.get("experts")) and _positive_int(r.get("top"))
                and _number(r.get("scale"))):
            yield f"{where}.mlp.router needs positive integers 'experts' and 'top' and a number 'scale', found {r!r}"
            return
        if r["top"] > r["experts"]:
            yield f"{where}.mlp.router.top={r['top']} exceeds its {r['experts']} experts"
        g = r.get("groups")
        if g is not None:
            if not (isinstance(g, dict) and _positive_int(g.get("count")) and _positive_int(g.get("keep"))
                    and g["keep"] <= g["count"]):
                yield f"{where}.mlp.router.groups needs 'count' >= 'keep' >= 1, found {g!r}"
            elif r["experts"] % g["count"]:
                yield f"{where}.mlp.router: {r['experts']} experts do not form {g['count']} equal groups"
            elif r["top"] > g["keep"] * (r["experts"] // g["count"]):
                yield f"{where}.mlp.router: top={r['top']} exceeds the experts of {g['keep']} groups"

    # ---- derived -------------------------------------------------------
    def eos_token_ids(self) -> Tuple[int, ...]:
        return () if self.eos_token_id is None else (int(self.eos_token_id),)
