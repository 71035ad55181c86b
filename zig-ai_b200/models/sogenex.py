"""The Sogenex design as a list of layers made from parts.

The embedding rows get the sinusoidal vector of their position.  Every layer is a pre-norm residual block whose RMS norms keep
their weights around zero (`x / rms(x) * (1 + w)`); its mixer is a state-space recurrence with one decay per head (Mamba-2) or
windowed differential attention without rotation; its feed-forward, where it has one, is a mixture of experts down(relu(up)^2)
chosen by their logits, with a gated unit of the same form for every token.  A layer may run on an earlier layer's tensors with
a cache and state of its own.  After the final norm an untied head whose logits are scaled and capped.

Tensor names: `embed`, `head`, `final.norm`, and per layer i `l<i>.norm1`, `norm2`, `l<i>.mix.<tensor>` and `l<i>.mlp.router`,
`router.b`, `e<n>.up`, `e<n>.down`, `shared.up`, `shared.down`, `shared.sg`.
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.sogenex import ARCHITECTURE, SogenexConfig
from ..parts.base import LayerCall, LayerSpec, ModelSpec, PartSpec

MAMBA2_NAMES = {"in": "mix.in", "conv": "mix.conv", "conv_bias": "mix.conv.b", "dt_bias": "mix.dt_bias", "a_log": "mix.A_log",
                "d": "mix.D", "norm": "mix.norm", "o": "mix.o"}
ATTENTION_NAMES = {k: f"mix.{k}" for k in ("q", "k", "v", "o", "lq1", "lk1", "lq2", "lk2")}
EXPERT_NAMES = {"router": "mlp.router", "router_bias": "mlp.router.b", "up": "mlp.e{e}.up", "down": "mlp.e{e}.down",
                "shared_gate": "mlp.shared.sg"}
SHARED_NAMES = {"up": "mlp.shared.up", "down": "mlp.shared.down"}
NORM_OFFSET = 1.0           # the design's norms multiply by 1 + the stored weight
POSITION_BASE = 10000.0     # of the sinusoidal position vectors


def mixer_spec(cfg: SogenexConfig, kind: str, m: dict) -> PartSpec:
    W, eps = cfg.width, cfg.norm_eps
    if kind == "mamba2":
        return PartSpec("mamba2", dict(hidden=W, heads=m["heads"], vdim=m["vdim"], state=m["state"], groups=m["groups"], taps=m["conv"],
                                       norm_parts=m["norm_groups"], eps=eps, names=MAMBA2_NAMES))
    return PartSpec("attention", dict(
        hidden=W, heads=m["heads"], kv_heads=m["kv_heads"], head_dim=m["dim"], value_dim=m["vdim"], qk_norm=False, eps=eps,
        position=PartSpec("none", {}), window=m["mask"]["size"], scale=m["scale"], differential={"diff": m["diff"]}, names=ATTENTION_NAMES))


def feed_forward_spec(cfg: SogenexConfig, mlp: dict) -> PartSpec:
    shared = None
    if mlp["shared"] is not None:
        shared = PartSpec("dense", dict(hidden=cfg.width, ff_dim=mlp["shared"]["ff"], activation="relu2", names=SHARED_NAMES))
    return PartSpec("routed_experts", dict(
        hidden=cfg.width, ff_dim=mlp["expert"]["ff"], experts=mlp["router"]["experts"], top=mlp["router"]["top"], weight_on="output",
        score="chosen", router_bias=True, expert_act="relu2", shared=shared, shared_gate=shared is not None, names=EXPERT_NAMES))


def build_spec(cfg: SogenexConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps
    norm = lambda name: PartSpec("rmsnorm", dict(size=W, eps=eps, weight=name, offset=NORM_OFFSET))
    layers, order, spec_of = [], [], {}
    for i, layer in enumerate(cfg.layers):
        if "weights_of" in layer:
            # the earlier layer's block runs once more; this entry of the running order has a cache and state of its own
            spec_of[i] = spec_of[layer["weights_of"]]
            order.append(LayerCall(spec_of[i]))
            continue
        block = dict(mixer=mixer_spec(cfg, layer["type"], layer["mixer"]), mixer_norm=norm("norm1"))
        if layer["mlp"] is not None:
            block.update(feed_forward=feed_forward_spec(cfg, layer["mlp"]), ff_norm=norm("norm2"))
        spec_of[i] = len(layers)
        layers.append(LayerSpec(prefix=f"l{i}.", block=PartSpec("prenorm_residual", block)))
        order.append(LayerCall(spec_of[i]))
    return ModelSpec(
        architecture=ARCHITECTURE, hidden_size=W, vocab_size=cfg.vocab, max_positions=cfg.max_positions,
        embedding=PartSpec("embedding", dict(weight="embed", sinusoidal=POSITION_BASE)),
        layers=layers, order=order, final_norm=norm("final.norm"),
        head=PartSpec("linear_head", dict(weight="head", tied=False, scale=cfg.logit_scale, softcap=cfg.logit_softcap)))


register_architecture(ARCHITECTURE, SogenexConfig, build_spec, replace=True)
