"""Configuration of the Pirozen design, read from its own config.json keys.

    architecture      "Pirozen"
    vocab, width      vocabulary and model width
    norm.eps          eps of every RMS norm (inside the root)
    token_side.dim    entries that every layer takes from a token's side row (absent or null: no such term)
    loop              {start, stop, times}: layers start .. stop-1 run `times` times in a row (absent or null: no loop)
    layers            one entry per layer: `type` (which mixer), `mixer` (its sizes and constants), `mlp` (null, or {kind: "moe",
                      expert: {ff}, router: {experts, identity, top, scale, groups: {count, keep} or null}, shared: {ff} or null})

Mixers by `type`:
    attention     heads, kv_heads, dim, vdim, scale, mask {size}, rot {base, dims, scaling: {factor, original, fast, slow} or null}
Every size and constant comes from the file; nothing is assumed equal to anything else.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .base import ConfigError, ModelConfig, read_key

ARCHITECTURE = "Pirozen"
MAX_POSITIONS = 1 << 20      # the design names no limit; block tables and graphs are sized by the cache, not by this
MIXERS = ("attention",)


def _object(d, key, where, required=True):
    v = d.get(key) if isinstance(d, dict) else None
    if v is None and not required:
        return None
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: required key '{key}' should be an object")
    return v


def _sizes(m, names, where, least=1):
    out = {k: read_key(m, k, int, where=where) for k in names}
    for k, v in out.items():
        if v < least:
            raise ConfigError(f"{where}: '{k}' should be at least {least}, got {v}")
    return out


def _rotation(rot, dim, where):
    out = {"base": read_key(rot, "base", float, where=where), "dims": read_key(rot, "dims", int, where=where), "scaling": None}
    if out["base"] <= 1.0 or out["dims"] % 2 or not 0 <= out["dims"] <= dim:
        raise ConfigError(f"{where}: base should be above 1, dims even and at most the head's {dim}")
    sc = _object(rot, "scaling", where, required=False)
    if sc is not None:
        out["scaling"] = {k: read_key(sc, k, float, where=where + ".scaling") for k in ("factor", "original", "fast", "slow")}
        if min(out["scaling"].values()) <= 0:
            raise ConfigError(f"{where}.scaling: factor, original, fast and slow should be positive")
    return out


def _attention(m, where):
    out = _sizes(m, ("heads", "kv_heads", "dim", "vdim"), where)
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"{where}: heads should be a multiple of kv_heads")
    out["scale"] = read_key(m, "scale", float, where=where)
    out["mask"] = _sizes(_object(m, "mask", where), ("size",), where + ".mask")
    out["rot"] = _rotation(_object(m, "rot", where), out["dim"], where + ".rot")
    return out


def _mlp(mlp, where):
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"{where} should be an object or null")
    kind = read_key(mlp, "kind", str, where=where)
    if kind != "moe":
        raise ConfigError(f"{where}: unknown kind '{kind}'; known: moe")
    r, at = _object(mlp, "router", where), where + ".router"
    router = _sizes(r, ("experts", "top"), at)
    router["identity"] = read_key(r, "identity", int, default=0, where=at)
    router["scale"] = read_key(r, "scale", float, default=1.0, where=at)
    total = router["experts"] + router["identity"]
    if router["identity"] < 0 or router["top"] > total:
        raise ConfigError(f"{at}: identity should not be negative, top at most experts + identity")
    groups = _object(r, "groups", at, required=False)
    router["groups"] = None
    if groups is not None:
        g = router["groups"] = _sizes(groups, ("count", "keep"), at + ".groups")
        if total % g["count"] or g["keep"] > g["count"] or g["keep"] * (total // g["count"]) < router["top"]:
            raise ConfigError(f"{at}.groups: experts and identities should form equal groups, of which those kept hold at least top")
    shared = _object(mlp, "shared", where, required=False)
    return {"kind": kind, "expert": _sizes(_object(mlp, "expert", where), ("ff",), where + ".expert"), "router": router,
            "shared": None if shared is None else _sizes(shared, ("ff",), where + ".shared")}


@dataclass
class PirozenConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm_eps: float = 1e-6
    token_side: Optional[int] = None
    loop: Optional[Dict[str, int]] = None
    layers: List[Dict[str, Any]] = field(default_factory=list)
    max_positions: int = MAX_POSITIONS

    # the names the engine and the command line use for every architecture
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def max_position_embeddings(self) -> int:
        return self.max_positions

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "PirozenConfig":
        vocab, width = read_key(d, "vocab", int), read_key(d, "width", int)
        if vocab < 1 or width < 1:
            raise ConfigError("vocab and width should be positive")
        layers_in = read_key(d, "layers", list)
        if not layers_in:
            raise ConfigError("'layers' should list at least one layer")
        layers, readers = [], {"attention": _attention}
        for i, entry in enumerate(layers_in):
            where = f"layers[{i}]"
            if not isinstance(entry, dict):
                raise ConfigError(f"{where} should be an object")
            kind = read_key(entry, "type", str, where=where)
            if kind not in readers:
                raise ConfigError(f"{where}: unknown mixer type '{kind}'; known: {', '.join(MIXERS)}")
            layers.append({"type": kind, "mixer": readers[kind](_object(entry, "mixer", where), where + ".mixer"),
                           "mlp": _mlp(entry.get("mlp"), where + ".mlp")})
        side = _object(d, "token_side", "config.json", required=False)
        loop = _object(d, "loop", "config.json", required=False)
        if loop is not None:
            loop = {"start": read_key(loop, "start", int, where="loop"), **_sizes(loop, ("stop", "times"), "loop")}
            if not 0 <= loop["start"] < loop["stop"] <= len(layers):
                raise ConfigError("loop: start .. stop-1 should be layers of the model, at least one")
        return cls(ARCHITECTURE, vocab=vocab, width=width, norm_eps=read_key(_object(d, "norm", "config.json"), "eps", float, where="norm"),
                   token_side=None if side is None else _sizes(side, ("dim",), "token_side")["dim"], loop=loop, layers=layers,
                   max_positions=read_key(d, "max_positions", int, default=MAX_POSITIONS))

    def to_dict(self) -> Dict[str, Any]:
        out = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "layers": copy.deepcopy(self.layers)}
        if self.token_side is not None:
            out["token_side"] = {"dim": self.token_side}
        if self.loop is not None:
            out["loop"] = dict(self.loop)
        if self.max_positions != MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        return out
