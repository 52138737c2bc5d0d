"""GoridraConfig: the sizes and constants of a Goridra decoder, read from config.json.

config.json of this design:
    architecture    "Goridra"
    vocab, width    sizes of the embedding table, which is also the head
    norm.eps        the epsilon of every layer norm
    logit_softcap   optional: a cap on the logits
    layers          a list; each entry has `type` ("attention"), `mixer` and `mlp` (an object or null)
      mixer         heads, kv_heads, dim, vdim, scale; optional mask {size} (chunks of that many positions), rot
                    {dims, base}, kv_from (the index of an earlier layer with keys and values of its own, which this
                    layer reads instead of projecting any)
      mlp           kind "dense", ff; or kind "moe", expert {ff}, router {experts, top, optional groups {count, keep}}
Every key below the top level is checked and an unknown one is refused: it would be a mechanism this code does not
have.  Top-level keys beyond these are a file's own notes.  The design has no largest position and no stop tokens.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass

from .base import ConfigError, _Reader
from .fovirax import _obj, _only


def _attention(raw, what, index: int, done: list) -> dict:
    raw = _obj(raw, what)
    _only(raw, what, ("heads", "kv_heads", "dim", "vdim", "scale", "mask", "rot", "kv_from"))
    r = _Reader(raw)
    m = {"heads": r.integer("heads"), "kv_heads": r.integer("kv_heads"), "dim": r.integer("dim"),
         "vdim": r.integer("vdim"), "scale": r.number("scale"), "mask": None, "rot": None, "kv_from": None}
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"config.json: `{what}`: heads {m['heads']} is not a multiple of kv_heads {m['kv_heads']}")
    if raw.get("mask") is not None:
        mask = _obj(raw["mask"], what + ".mask")
        _only(mask, what + ".mask", ("size",))
        m["mask"] = {"size": _Reader(mask).integer("size")}
    if raw.get("rot") is not None:
        rot = _obj(raw["rot"], what + ".rot")
        _only(rot, what + ".rot", ("dims", "base"))
        rr = _Reader(rot)
        dims, base = rr.integer("dims", minimum=0), rr.number("base")
        if dims % 2 or dims > m["dim"]:
            raise ConfigError(f"config.json: `{what}.rot.dims` must be even and at most the head's dim {m['dim']}")
        if dims:
            m["rot"] = {"dims": dims, "base": base}
    src = r.integer("kv_from", required=False, minimum=0)
    if src is not None:
        if src >= index or done[src]["mixer"]["kv_from"] is not None:
            raise ConfigError(f"config.json: `{what}.kv_from` must name an earlier layer with keys and values of its "
                              f"own, got {src}")
        owner = done[src]["mixer"]
        for key in ("kv_heads", "dim", "vdim", "rot"):
            if owner[key] != m[key]:
                raise ConfigError(f"config.json: `{what}.kv_from`: layer {src} has {key} {owner[key]}, this layer {m[key]}")
        m["kv_from"] = src
    return m


def _mlp(raw, what):
    if raw is None:
        return None
    raw = _obj(raw, what)
    kind = raw.get("kind")
    if kind == "dense":
        _only(raw, what, ("kind", "ff"))
        return {"kind": "dense", "ff": _Reader(raw).integer("ff")}
    if kind != "moe":
        raise ConfigError(f"config.json: `{what}.kind` must be \"dense\" or \"moe\", got {kind!r}")
    _only(raw, what, ("kind", "expert", "router"))
    expert, router = _obj(raw.get("expert"), what + ".expert"), _obj(raw.get("router"), what + ".router")
    _only(expert, what + ".expert", ("ff",))
    _only(router, what + ".router", ("experts", "top", "groups"))
    rr = _Reader(router)
    experts, top, groups = rr.integer("experts"), rr.integer("top"), None
    reach = experts
    if router.get("groups") is not None:
        g = _obj(router["groups"], what + ".router.groups")
        _only(g, what + ".router.groups", ("count", "keep"))
        groups = {"count": _Reader(g).integer("count"), "keep": _Reader(g).integer("keep")}
        if experts % groups["count"] or groups["keep"] > groups["count"]:
            raise ConfigError(f"config.json: `{what}.router.groups`: {experts} experts do not stand in {groups['count']} "
                              f"equal groups of which {groups['keep']} stay")
        reach = groups["keep"] * (experts // groups["count"])
    if top > reach:
        raise ConfigError(f"config.json: `{what}.router`: top {top} exceeds the {reach} experts that can be chosen")
    return {"kind": "moe", "expert": {"ff": _Reader(expert).integer("ff")},
            "router": {"experts": experts, "top": top, "groups": groups}}


@dataclass(frozen=True)
class GoridraConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    logit_softcap: float | None
    layers: tuple              # of {"type", "mixer", "mlp"} with checked contents

    @staticmethod
    def from_dict(raw: dict) -> "GoridraConfig":
        r = _Reader(raw)
        norm = _obj(raw.get("norm"), "norm")
        _only(norm, "norm", ("eps",))
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: `layers` must be a list with at least one layer")
        out: list = []
        for i, layer in enumerate(layers):
            what = f"layers[{i}]"
            layer = _obj(layer, what)
            _only(layer, what, ("type", "mixer", "mlp"))
            if layer.get("type") != "attention":
                raise ConfigError(f"config.json: `{what}.type` must be \"attention\", got {layer.get('type')!r}")
            out.append({"type": "attention", "mixer": _attention(layer.get("mixer"), what + ".mixer", i, out),
                        "mlp": _mlp(layer.get("mlp"), what + ".mlp")})
        name = raw.get("architecture") or (raw.get("architectures") or ["Goridra"])[0]
        return GoridraConfig(architecture=name, vocab=r.integer("vocab"), width=r.integer("width"),
                             norm_eps=_Reader(norm).number("eps"),
                             logit_softcap=r.number("logit_softcap", required=False), layers=tuple(out))

    def to_dict(self) -> dict:
        """The config.json that `from_dict` reads back to an equal configuration."""
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "layers": copy.deepcopy(list(self.layers))}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        return d
