"""The Pirozen design as a list of layers made from parts.

Every layer is a parallel residual block: windowed grouped-query attention (biases on all four projections, a norm per head of
queries and keys, a partial rotation with frequencies stretched for long contexts, a sigmoid gate per head) and a mixture of
experts read the same stream through a norm each and are added to it together; then a term from the layer's part of the
token's row in a side table joins, behind a norm of its own.  Experts are chosen by softmax score plus a learned correction out of
the best groups, some of the router's outputs stand for the input itself, and one more expert runs for every token.  A run of
layers may be passed several times in a row, each time with caches of its own and behind a product of the stream and the
embedding's output.  Final norm, untied head.

Tensor names: `embed`, `side.embed`, `loop.in`, `head`, `final.norm`, and per layer i `l<i>.norm1`, `norm2`, `l<i>.mix.<tensor>`
(a bias: the tensor's name + `.b`, a norm's weight + `.norm`), `l<i>.mlp.router`, `correction`, `e<n>.gate`, `up`, `down`,
`shared.gate`, `up`, `down`, and `l<i>.side.gate`, `proj`, `norm`.
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.pirozen import ARCHITECTURE, PirozenConfig
from ..parts.base import LayerCall, LayerSpec, ModelSpec, PartSpec

ATTENTION_NAMES = {"q": "mix.q", "k": "mix.k", "v": "mix.v", "o": "mix.o", "g": "mix.g", "q_bias": "mix.q.b", "k_bias": "mix.k.b",
                   "v_bias": "mix.v.b", "o_bias": "mix.o.b", "q_norm": "mix.q.norm", "k_norm": "mix.k.norm"}
EXPERT_NAMES = {"router": "mlp.router", "correction": "mlp.correction", "gate": "mlp.e{e}.gate", "up": "mlp.e{e}.up",
                "down": "mlp.e{e}.down"}
SHARED_NAMES = {"gate": "mlp.shared.gate", "up": "mlp.shared.up", "down": "mlp.shared.down"}
SIDE_NAMES = {"gate": "side.gate", "proj": "side.proj", "norm": "side.norm"}


def mixer_spec(cfg: PirozenConfig, m: dict) -> PartSpec:
    rot = m["rot"]
    position = PartSpec("none", {})
    if rot["dims"]:
        position = PartSpec("rotary_half_split", dict(head_dim=m["dim"], theta=rot["base"], rotary_dim=rot["dims"], scaling=rot["scaling"]))
    return PartSpec("attention", dict(
        hidden=cfg.width, heads=m["heads"], kv_heads=m["kv_heads"], head_dim=m["dim"], value_dim=m["vdim"], qk_norm=True,
        eps=cfg.norm_eps, position=position, window=m["mask"]["size"], scale=m["scale"], bias=True, out_bias=True, gate="head",
        names=ATTENTION_NAMES))


def feed_forward_spec(cfg: PirozenConfig, mlp: dict) -> PartSpec:
    r, shared = mlp["router"], None
    if mlp["shared"] is not None:
        shared = PartSpec("swiglu", dict(hidden=cfg.width, ff_dim=mlp["shared"]["ff"], names=SHARED_NAMES))
    return PartSpec("routed_experts", dict(
        hidden=cfg.width, ff_dim=mlp["expert"]["ff"], experts=r["experts"], top=r["top"], renormalize=True, weight_on="output",
        score="softmax", correction=True, groups=r["groups"], identities=r["identity"], weight_scale=r["scale"], shared=shared,
        names=EXPERT_NAMES))


def running_order(n_layers: int, loop, merge: int):
    """The layers' entries with the repeated ones written out, each pass behind an entry of layer `merge`."""
    if loop is None:
        return [LayerCall(i) for i in range(n_layers)]
    inner = [merge] + list(range(loop["start"], loop["stop"]))
    return [LayerCall(i) for i in list(range(loop["start"])) + inner * loop["times"] + list(range(loop["stop"], n_layers))]


def build_spec(cfg: PirozenConfig) -> ModelSpec:
    W, eps, side = cfg.width, cfg.norm_eps, cfg.token_side
    norm = lambda name: PartSpec("rmsnorm", dict(size=W, eps=eps, weight=name))
    layers, tables = [], {}
    if side is not None:
        tables["side"] = PartSpec("token_table", dict(weight="side.embed", columns=side * len(cfg.layers)))
    for i, layer in enumerate(cfg.layers):
        block = dict(mixer=mixer_spec(cfg, layer["mixer"]), mixer_norm=norm("norm1"))
        if layer["mlp"] is not None:
            block.update(feed_forward=feed_forward_spec(cfg, layer["mlp"]), ff_norm=norm("norm2"))
        if side is not None:
            block["token_input"] = PartSpec("side_rows", dict(hidden=W, dim=side, at=i * side, eps=eps, table="side", names=SIDE_NAMES))
        layers.append(LayerSpec(prefix=f"l{i}.", block=PartSpec("parallel_residual", block)))
    order = running_order(len(layers), cfg.loop, merge=len(layers))
    if cfg.loop is not None:
        layers.append(LayerSpec(prefix="loop.", block=PartSpec("stream_merge", dict(hidden=W, weight="in"))))
    return ModelSpec(
        architecture=ARCHITECTURE, hidden_size=W, vocab_size=cfg.vocab, max_positions=cfg.max_positions,
        embedding=PartSpec("embedding", dict(weight="embed")), layers=layers, order=order, final_norm=norm("final.norm"),
        head=PartSpec("linear_head", dict(weight="head", tied=False)), tables=tables)


register_architecture(ARCHITECTURE, PirozenConfig, build_spec, replace=True)
