"""Configuration of the Sogenex design, read from its own config.json keys.

    architecture      "Sogenex"
    vocab, width      vocabulary and model width
    norm.eps          eps of every RMS norm (inside the root)
    logit_scale       factor on the head's product
    logit_softcap     bound of the scaled logits: cap tanh(logits / cap)
    layers            one entry per layer: `type` (which mixer), `mixer` (its sizes and constants), `mlp` (null, or {kind: "moe",
                      expert: {ff}, router: {experts, top}, shared: {ff} or null}), and optionally `weights_of` (an earlier
                      layer whose tensors this one uses; type, mixer and mlp equal that layer's)

Mixers by `type`:
    mamba2        heads, vdim, state, groups, conv (taps), norm_groups
    attention     heads, kv_heads, dim (of one map's query and key), vdim, scale, mask {size}, diff
Every size and constant comes from the file; nothing is assumed equal to anything else.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .base import ConfigError, ModelConfig, read_key

ARCHITECTURE = "Sogenex"
MAX_POSITIONS = 1 << 20      # the design names no limit; block tables and graphs are sized by the cache, not by this
MIXERS = ("mamba2", "attention")


def _object(d, key, where, required=True):
    v = d.get(key) if isinstance(d, dict) else None
    if v is None and not required:
        return None
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: required key '{key}' should be an object")
    return v


def _sizes(m, names, where):
    out = {k: read_key(m, k, int, where=where) for k in names}
    for k, v in out.items():
        if v < 1:
            raise ConfigError(f"{where}: '{k}' should be at least 1, got {v}")
    return out


def _mamba2(m, where):
    out = _sizes(m, ("heads", "vdim", "state", "groups", "conv", "norm_groups"), where)
    if out["heads"] % out["groups"]:
        raise ConfigError(f"{where}: heads should be a multiple of groups")
    if (out["heads"] * out["vdim"]) % out["norm_groups"]:
        raise ConfigError(f"{where}: heads * vdim should be a multiple of norm_groups")
    return out


def _attention(m, where):
    out = _sizes(m, ("heads", "kv_heads", "dim", "vdim"), where)
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"{where}: heads should be a multiple of kv_heads")
    out["scale"], out["diff"] = read_key(m, "scale", float, where=where), read_key(m, "diff", float, where=where)
    out["mask"] = _sizes(_object(m, "mask", where), ("size",), where + ".mask")
    return out


def _mlp(mlp, where):
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"{where} should be an object or null")
    kind = read_key(mlp, "kind", str, where=where)
    if kind != "moe":
        raise ConfigError(f"{where}: unknown kind '{kind}'; known: moe")
    out = {"kind": kind, "expert": _sizes(_object(mlp, "expert", where), ("ff",), where + ".expert"),
           "router": _sizes(_object(mlp, "router", where), ("experts", "top"), where + ".router")}
    if out["router"]["top"] > out["router"]["experts"]:
        raise ConfigError(f"{where}: router.top should be at most router.experts")
    shared = _object(mlp, "shared", where, required=False)
    out["shared"] = None if shared is None else _sizes(shared, ("ff",), where + ".shared")
    return out


@dataclass
class SogenexConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm_eps: float = 1e-6
    logit_scale: float = 1.0
    logit_softcap: Optional[float] = None
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
    def from_dict(cls, d: Dict[str, Any]) -> "SogenexConfig":
        vocab, width = read_key(d, "vocab", int), read_key(d, "width", int)
        if vocab < 1 or width < 1:
            raise ConfigError("vocab and width should be positive")
        layers_in = read_key(d, "layers", list)
        if not layers_in:
            raise ConfigError("'layers' should list at least one layer")
        layers, readers = [], {"mamba2": _mamba2, "attention": _attention}
        for i, entry in enumerate(layers_in):
            where = f"layers[{i}]"
            if not isinstance(entry, dict):
                raise ConfigError(f"{where} should be an object")
            kind = read_key(entry, "type", str, where=where)
            if kind not in readers:
                raise ConfigError(f"{where}: unknown mixer type '{kind}'; known: {', '.join(MIXERS)}")
            layer = {"type": kind, "mixer": readers[kind](_object(entry, "mixer", where), where + ".mixer"),
                     "mlp": _mlp(entry.get("mlp"), where + ".mlp")}
            if entry.get("weights_of") is not None:
                src = read_key(entry, "weights_of", int, where=where)
                if not 0 <= src < i:
                    raise ConfigError(f"{where}: weights_of should name an earlier layer")
                if {k: v for k, v in layers[src].items() if k != "weights_of"} != layer:
                    raise ConfigError(f"{where}: a layer that uses layer {src}'s tensors should equal it in type, mixer and mlp")
                layer["weights_of"] = layers[src].get("weights_of", src)
            layers.append(layer)
        softcap = read_key(d, "logit_softcap", float, default=None)
        if softcap is not None and softcap <= 0:
            raise ConfigError("logit_softcap should be positive")
        return cls(ARCHITECTURE, vocab=vocab, width=width, norm_eps=read_key(_object(d, "norm", "config.json"), "eps", float, where="norm"),
                   logit_scale=read_key(d, "logit_scale", float, default=1.0), logit_softcap=softcap, layers=layers,
                   max_positions=read_key(d, "max_positions", int, default=MAX_POSITIONS))

    def to_dict(self) -> Dict[str, Any]:
        out = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "logit_scale": self.logit_scale, "logit_softcap": self.logit_softcap, "layers": copy.deepcopy(self.layers)}
        if self.max_positions != MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        return out
