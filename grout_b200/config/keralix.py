"""Configuration of the Keralix decoder.

The file names the design under ``architecture`` and describes the model layer by layer:
``layers`` is a list of objects ``{"type", "mixer", "mlp"}`` (``mlp`` null: the layer has
no feed-forward).  Nothing that the arithmetic needs is defaulted; a rotation, a window and
a cap of the scores may be absent, and the ranks of the low-rank gates of a
``channel_delta`` mixer are those of its tensors.

    vocab, width                  sizes of the embedding table (which is the head, too) and of a stream
    streams                       residual streams that run side by side
    embedding.scale               factor of the embedded token
    norm.eps                      epsilon of every RMS norm
    layers[i].type                "attention" | "latent_attention" | "channel_delta"
    layers[i].mixer (attention)   heads, kv_heads, dim, vdim (the values are the keys: equal to dim),
                                  conv (taps), scale, softcap, rot.{base, dims}, mask.size
    layers[i].mixer (latent_attention)
                                  heads, dim, vdim, q_rank, kv_rank, scale
    layers[i].mixer (channel_delta)
                                  heads, kv_heads, dim, vdim, conv (taps)
    layers[i].mlp                 {"kind": "dense", "ff"}
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .base import ModelConfig

_SIZES = {"attention": ("heads", "kv_heads", "dim", "vdim", "conv"),
          "latent_attention": ("heads", "dim", "vdim", "q_rank", "kv_rank"),
          "channel_delta": ("heads", "kv_heads", "dim", "vdim", "conv")}
MAX_STREAMS = 16


def _number(v) -> bool:
    return isinstance(v, (int, float)) and not isinstance(v, bool)


def _positive_int(v) -> bool:
    return isinstance(v, int) and not isinstance(v, bool) and v > 0


@dataclass(frozen=True)
class KeralixConfig(ModelConfig):
    vocab: int
    width: int
    streams: int
    layers: Tuple[dict, ...]
    norm: dict
    embedding: dict
    architecture: str = "Keralix"
    eos_token_id: Optional[int] = None

    def validate(self):
        for key in ("vocab", "width", "streams"):
            if not _positive_int(getattr(self, key)):
                yield f"'{key}' must be a positive integer, found {getattr(self, key)!r}"
        if _positive_int(self.streams) and self.streams > MAX_STREAMS:
            yield f"'streams'={self.streams}: at most {MAX_STREAMS} run side by side"
        if not _number(self.norm.get("eps")) or not self.norm["eps"] > 0:
            yield f"'norm.eps' must be a positive number, found {self.norm.get('eps')!r}"
        if not _number(self.embedding.get("scale")):
            yield f"'embedding.scale' must be a number, found {self.embedding.get('scale')!r}"
        if not self.layers:
            yield "'layers' is empty"
        for i, layer in enumerate(self.layers):
            yield from self._layer_problems(f"layers[{i}]", layer)

    def _layer_problems(self, where, layer):
        if not isinstance(layer, dict):
            yield f"{where} is not an object"
            return
        kind = layer.get("type")
        if kind not in _SIZES:
            yield f"{where}.type={kind!r}: this design has {sorted(_SIZES)}"
            return
        m = layer.get("mixer")
        if not isinstance(m, dict):
            yield f"{where}.mixer is missing"
            return
        bad = [k for k in _SIZES[kind] if not _positive_int(m.get(k))]
        for key in bad:
            yield f"{where}.mixer.{key} must be a positive integer, found {m.get(key)!r}"
        if bad:
            return
        if "kv_heads" in _SIZES[kind] and m["heads"] % m["kv_heads"]:
            yield f"{where}.mixer: {m['heads']} heads cannot share {m['kv_heads']} kv heads"
        if kind != "channel_delta" and not _number(m.get("scale")):
            yield f"{where}.mixer.scale must be a number, found {m.get('scale')!r}"
        if kind == "attention":
            yield from self._attention_problems(where + ".mixer", m)
        mlp = layer.get("mlp")
        if mlp is not None and not (isinstance(mlp, dict) and mlp.get("kind") == "dense"
                                    and _positive_int(mlp.get("ff"))):
            yield f"{where}.mlp must be null or {{'kind': 'dense', 'ff': rows}}, found {mlp!r}"

    def _attention_problems(self, where, m):
        if m["vdim"] != m["dim"]:
            yield f"{where}: the values are the keys, so vdim={m['vdim']} must equal dim={m['dim']}"
        cap = m.get("softcap")
        if cap is not None and not (_number(cap) and cap > 0):
            yield f"{where}.softcap must be a positive number, found {cap!r}"
        rot = m.get("rot")
        if rot is not None:
            dims = rot.get("dims") if isinstance(rot, dict) else None
            if not (isinstance(dims, int) and not isinstance(dims, bool) and dims >= 0 and dims % 2 == 0
                    and _number(rot.get("base")) and rot["base"] > 0):
                yield f"{where}.rot needs a positive 'base' and an even 'dims', found {rot!r}"
            elif dims > m["dim"]:
                yield f"{where}.rot.dims={dims} exceeds the head's {m['dim']} elements"
        mask = m.get("mask")
        if mask is not None and not (isinstance(mask, dict) and _positive_int(mask.get("size"))):
            yield f"{where}.mask needs a positive integer 'size', found {mask!r}"

    # ---- derived -------------------------------------------------------
    def eos_token_ids(self) -> Tuple[int, ...]:
        return () if self.eos_token_id is None else (int(self.eos_token_id),)
