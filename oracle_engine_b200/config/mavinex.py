"""MavinexConfig: the sizes and constants of a Mavinex decoder, read from config.json.

config.json of this design:
    architecture     "Mavinex"
    vocab, width     sizes of the embedding table and of the head
    embedding.scale  the constant an embedding row is multiplied by (default 1)
    norm.eps         the epsilon of every root mean square
    postln_alpha     the constant the stream is multiplied by before a sublayer's output joins it
    layers           a list; each entry has `type`, `mixer`, `mlp` (an object or null) and optionally
                     `weights_of` (the index of a layer whose tensors this one computes with; the rest of the entry
                     equals that layer's)
      "parallel"          mixer.left: heads, kv_heads, dim, vdim, scale; optional mask {size}, rot {dims, base, optional
                          scaling {factor, low, high, original}};  mixer.right: inner, state, dt_rank, conv
      "latent_attention"  mixer: heads, dim, rot_dim, vdim, kv_rank, scale; optional mask {size}, rot {dims, base,
                          optional scaling {factor, original, fast, slow}} (dims up to rot_dim)
      mlp                 kind "moe", expert {ff}, router {experts, top}
Every key below the top level is checked and an unknown one is refused: it would be a mechanism this code does not
have.  Top-level keys beyond these are a file's own notes.  The design has no largest position and no stop tokens.
"""
from __future__ import annotations

import copy
import math
from dataclasses import dataclass

from .base import ConfigError, _Reader
from .fovirax import _obj, _only, _rot


def _mask(raw, what):
    if raw is None:
        return None
    raw = _obj(raw, what)
    _only(raw, what, ("size",))
    return {"size": _Reader(raw).integer("size")}


def _yarn_rot(raw, what, dim):
    """None, or {"dims", "base", "scaling": None or {"factor", "original", "fast", "slow"}}."""
    if raw is None:
        return None
    raw = _obj(raw, what)
    rot = _rot({k: v for k, v in raw.items() if k != "scaling"}, what, dim)
    if rot is not None and raw.get("scaling") is not None:
        sc = _obj(raw["scaling"], what + ".scaling")
        _only(sc, what + ".scaling", ("factor", "original", "fast", "slow"))
        r = _Reader(sc)
        rot["scaling"] = {k: r.number(k) for k in ("factor", "original", "fast", "slow")}
        if not (math.isfinite(rot["base"]) and rot["base"] > 1.0):
            raise ConfigError(f"config.json: `{what}.base` must be above 1 for its scaling, got {rot['base']}")
    return rot


def _left(raw, what):
    raw = _obj(raw, what)
    _only(raw, what, ("heads", "kv_heads", "dim", "vdim", "scale", "mask", "rot"))
    r = _Reader(raw)
    m = {"heads": r.integer("heads"), "kv_heads": r.integer("kv_heads"), "dim": r.integer("dim"),
         "vdim": r.integer("vdim"), "scale": r.number("scale")}
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"config.json: `{what}`: heads {m['heads']} is not a multiple of kv_heads {m['kv_heads']}")
    m["mask"] = _mask(raw.get("mask"), what + ".mask")
    m["rot"] = _rot(raw.get("rot"), what + ".rot", m["dim"])
    return m


def _right(raw, what):
    raw = _obj(raw, what)
    keys = ("inner", "state", "dt_rank", "conv")
    _only(raw, what, keys)
    r = _Reader(raw)
    return {k: r.integer(k) for k in keys}


def _latent(raw, what):
    raw = _obj(raw, what)
    sizes = ("heads", "dim", "vdim", "kv_rank")
    _only(raw, what, sizes + ("rot_dim", "scale", "mask", "rot"))
    r = _Reader(raw)
    m = {k: r.integer(k) for k in sizes}
    m["rot_dim"] = r.integer("rot_dim", default=0, required=False, minimum=0)
    m["scale"] = r.number("scale")
    m["mask"] = _mask(raw.get("mask"), what + ".mask")
    m["rot"] = _yarn_rot(raw.get("rot"), what + ".rot", m["rot_dim"])
    return m


def _mixer(kind, raw, what):
    if kind == "latent_attention":
        return _latent(raw, what)
    raw = _obj(raw, what)
    _only(raw, what, ("left", "right"))
    return {"left": _left(raw.get("left"), what + ".left"), "right": _right(raw.get("right"), what + ".right")}


def _mlp(raw, what):
    if raw is None:
        return None
    raw = _obj(raw, what)
    if raw.get("kind") != "moe":
        raise ConfigError(f"config.json: `{what}.kind` must be \"moe\", got {raw.get('kind')!r}")
    _only(raw, what, ("kind", "expert", "router"))
    expert, router = _obj(raw.get("expert"), what + ".expert"), _obj(raw.get("router"), what + ".router")
    _only(expert, what + ".expert", ("ff",))
    _only(router, what + ".router", ("experts", "top"))
    rr = _Reader(router)
    experts, top = rr.integer("experts"), rr.integer("top")
    if top > experts:
        raise ConfigError(f"config.json: `{what}.router`: top {top} exceeds the {experts} experts")
    return {"kind": "moe", "expert": {"ff": _Reader(expert).integer("ff")}, "router": {"experts": experts, "top": top}}


@dataclass(frozen=True)
class MavinexConfig:
    architecture: str
    vocab: int
    width: int
    embedding_scale: float
    norm_eps: float
    postln_alpha: float
    layers: tuple              # of {"type", "mixer", "mlp", "weights_of"} with checked contents

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i computes with (itself without `weights_of`)."""
        return _owner(self.layers, i)

    @staticmethod
    def from_dict(raw: dict) -> "MavinexConfig":
        r = _Reader(raw)
        norm = _obj(raw.get("norm"), "norm")
        _only(norm, "norm", ("eps",))
        emb = _obj(raw["embedding"], "embedding") if raw.get("embedding") is not None else {}
        _only(emb, "embedding", ("scale",))
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: `layers` must be a list with at least one layer")
        out: list = []
        for i, layer in enumerate(layers):
            what = f"layers[{i}]"
            layer = _obj(layer, what)
            _only(layer, what, ("type", "mixer", "mlp", "weights_of"))
            kind = layer.get("type")
            if kind not in ("parallel", "latent_attention"):
                raise ConfigError(f"config.json: `{what}.type` must be \"parallel\" or \"latent_attention\", got {kind!r}")
            src = _Reader(layer).integer("weights_of", required=False, minimum=0)
            if src is not None and src >= len(layers):
                raise ConfigError(f"config.json: `{what}.weights_of` names layer {src}, there are {len(layers)}")
            out.append({"type": kind, "mixer": _mixer(kind, layer.get("mixer"), what + ".mixer"),
                        "mlp": _mlp(layer.get("mlp"), what + ".mlp"), "weights_of": src})
        for i, layer in enumerate(out):
            j = _owner(out, i)
            if any(layer[k] != out[j][k] for k in ("type", "mixer", "mlp")):
                raise ConfigError(f"config.json: `layers[{i}]` differs from layer {j}, whose tensors it uses")
        name = raw.get("architecture") or (raw.get("architectures") or ["Mavinex"])[0]
        return MavinexConfig(architecture=name, vocab=r.integer("vocab"), width=r.integer("width"),
                             embedding_scale=_Reader(emb).number("scale", default=1.0, required=False),
                             norm_eps=_Reader(norm).number("eps"), postln_alpha=r.number("postln_alpha"),
                             layers=tuple(out))

    def to_dict(self) -> dict:
        """The config.json that `from_dict` reads back to an equal configuration."""
        layers = []
        for layer in copy.deepcopy(list(self.layers)):
            if layer["weights_of"] is None:
                del layer["weights_of"]
            layers.append(layer)
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.norm_eps},
                "postln_alpha": self.postln_alpha, "layers": layers}


def _owner(layers, i: int) -> int:
    seen = set()
    while layers[i]["weights_of"] is not None:
        if i in seen:
            raise ConfigError(f"config.json: `layers[{i}].weights_of` leads back to itself")
        seen.add(i)
        i = layers[i]["weights_of"]
    return i
