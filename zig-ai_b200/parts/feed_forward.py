"""SwiGLU feed-forward: `down( silu(gate(x)) * up(x) )`, no biases
(src/transformer/ffn.zig:7-34; device activation src/cuda/layer_kernels.cu:62-70; tensor names
src/transformer/hybrid_layer.zig:313-321).  The gate and up matrices are stacked into one
[2F, hidden] matrix at load so that one product feeds the activation.
"""
from __future__ import annotations

import torch

from .base import FeedForward, ParamDecl, make_part, register_part


class SwiGlu(FeedForward):
    """`names` gives the three tensors' names (gate, up, down).  `activation`: what the gate passes, silu by default, or
    one of gelu (erf), gelu_tanh, relu: `down( act(gate(x)) * up(x) )`."""
    accepts_lazy_input = True     # x goes straight into a product
    graph_safe = True      # forward launches kernels only; nothing is read back to the host
    kernel_libs = ("gemm_tc_pair",)       # gate/up products of many rows with the activation as their epilogue (bfloat16)

    def __init__(self, hidden: int, ff_dim: int, names=None, activation: str = "silu"):
        self.hidden, self.ff_dim, self.activation = int(hidden), int(ff_dim), str(activation)
        if self.activation not in ("silu", "gelu", "gelu_erf", "gelu_tanh", "relu"):
            raise ValueError(f"unknown activation '{self.activation}'")
        self.names = {"gate": "ffn_gate.weight", "up": "ffn_up.weight", "down": "ffn_down.weight", **(names or {})}

    def params(self):
        nm = self.names
        return {
            nm["gate"]: ParamDecl((self.ff_dim, self.hidden)),
            nm["up"]: ParamDecl((self.ff_dim, self.hidden)),
            nm["down"]: ParamDecl((self.hidden, self.ff_dim)),
        }

    def bind(self, tensors, dtype):
        nm = self.names
        self.w_gate_up = torch.cat([tensors[nm["gate"]], tensors[nm["up"]]], dim=0).contiguous()
        self.w_down = tensors[nm["down"]]
        self.dtype = dtype

    def forward(self, x, step):
        ops = step.ops
        if self.activation == "silu":
            a = ops.linear_swiglu(x, self.w_gate_up, self.ff_dim)
        else:
            a = ops.linear_glu(x, self.w_gate_up, self.ff_dim, self.activation)
        return ops.linear(a, self.w_down)


class DenseMlp(FeedForward):
    """`down( act(up(x)) )`, no gate and no biases; `activation` is one of gelu (the exact one, with erf),
    gelu_tanh, silu, relu, relu2 (the square of relu).  `names` gives the two tensors' names."""
    accepts_lazy_input = True     # x goes straight into a product
    graph_safe = True

    def __init__(self, hidden: int, ff_dim: int, activation: str = "gelu", names=None):
        self.hidden, self.ff_dim, self.activation = int(hidden), int(ff_dim), str(activation)
        if self.activation not in ("gelu", "gelu_erf", "gelu_tanh", "silu", "relu", "relu2"):
            raise ValueError(f"unknown activation '{self.activation}'")
        self.names = {"up": "ffn_up.weight", "down": "ffn_down.weight", **(names or {})}

    def params(self):
        return {self.names["up"]: ParamDecl((self.ff_dim, self.hidden)),
                self.names["down"]: ParamDecl((self.hidden, self.ff_dim))}

    def bind(self, tensors, dtype):
        self.w_up, self.w_down = tensors[self.names["up"]], tensors[self.names["down"]]
        self.dtype = dtype

    def forward(self, x, step):
        ops = step.ops
        return ops.linear(ops.linear_activation(x, self.w_up, self.activation), self.w_down)


class ClampedGlu(FeedForward):
    """A gated feed-forward with bounded branches, no biases:

        g = min(gate(x), limit);  u = clamp(up(x), -limit, limit);  out = down( g * sigmoid(alpha * g) * (u + 1) )

    The gate and up matrices are stacked into one [2F, hidden] matrix at load.  `names` gives the tensors' names."""
    accepts_lazy_input = True
    graph_safe = True

    def __init__(self, hidden: int, ff_dim: int, limit: float, alpha: float = 1.702, names=None):
        self.hidden, self.ff_dim, self.limit, self.alpha = int(hidden), int(ff_dim), float(limit), float(alpha)
        self.names = {"gate": "ffn_gate.weight", "up": "ffn_up.weight", "down": "ffn_down.weight", **(names or {})}

    def params(self):
        nm = self.names
        return {nm["gate"]: ParamDecl((self.ff_dim, self.hidden)), nm["up"]: ParamDecl((self.ff_dim, self.hidden)),
                nm["down"]: ParamDecl((self.hidden, self.ff_dim))}

    def bind(self, tensors, dtype):
        nm = self.names
        self.w_gate_up = torch.cat([tensors[nm["gate"]], tensors[nm["up"]]], dim=0).contiguous()
        self.w_down = tensors[nm["down"]]
        self.dtype = dtype

    def forward(self, x, step):
        ops = step.ops
        return ops.linear(ops.linear_clamped_glu(x, self.w_gate_up, self.ff_dim, self.limit, self.alpha), self.w_down)


class RoutedExperts(FeedForward):
    """A mixture of `experts` small SwiGLU feed-forwards, of which every token uses `top`:

        s = sigmoid(x . Wr^T)                 router, 32-bit
        chosen = the `top` experts with the largest s;   w_e = s_e   (divided by their sum with `renormalize`)
        out = sum over chosen e of  down_e( silu(gate_e(w_e x)) * up_e(w_e x) )          weight_on="input"
                                or  w_e down_e( silu(gate_e(x)) * up_e(x) )              weight_on="output"

    Experts have no biases.  The router's matrix is kept in 32-bit.  `names`: "router", and "gate", "up", "down" with
    `{e}` standing for the expert's number.

    Options: `score="softmax"` (s = softmax of the router's logits over all experts; with `renormalize` the chosen scores
    are divided by their sum + 1e-20); `expert_act="clamped"` with `limit` and `alpha` (experts of the bounded form
    min(g, limit) sigmoid(alpha min(g, limit)) (clamp(u, -limit, limit) + 1)); `shared`, the `PartSpec` of a feed-forward
    that every token passes beside its experts (its tensors under its own names) and whose output is added.

    `score="chosen"`: the logits choose and the weights are the softmax over the chosen logits alone; `router_bias` adds a
    learned number per expert (name "router_bias") to the logits.  `expert_act="relu2"`: experts without a gate,
    down_e( relu(up_e(x))^2 ).  `shared_gate`: the shared feed-forward's output times sigmoid(x . w) with a learned row w (name
    "shared_gate"), computed in 32-bit with the router.

    Options of the choice (with sigmoid or softmax scores): `correction` (a learned number per expert, name "correction", is
    added to the scores for the choice alone); `groups` = {count, keep} (equal groups of neighbouring experts; only the experts
    of the `keep` groups with the largest choice values can be chosen); `identities` (that many further outputs of the router
    stand for experts without tensors whose output is x itself); `weight_scale` (a factor on the weights)."""
    accepts_lazy_input = False    # the router and the experts read the normed rows themselves
    graph_safe = True             # routing stays on the device: forward launches kernels only
    kernel_libs = ("moe", "gemm_tc")      # (gemm_tc: the grouped products of steps with many rows an expert, bfloat16)

    def __init__(self, hidden: int, ff_dim: int, experts: int, top: int, renormalize: bool = False, weight_on: str = "input",
                 names=None, score: str = "sigmoid", expert_act: str = "silu", limit: float = 0.0, alpha: float = 1.702, shared=None,
                 router_bias: bool = False, shared_gate: bool = False, correction: bool = False, groups=None, identities: int = 0,
                 weight_scale: float = 1.0):
        self.hidden, self.ff_dim, self.experts, self.top = int(hidden), int(ff_dim), int(experts), int(top)
        self.renormalize, self.weight_on = bool(renormalize), weight_on
        self.correction, self.identities, self.weight_scale = bool(correction), int(identities), float(weight_scale)
        self.outputs = self.experts + self.identities                # what the router scores
        self.groups = None if groups is None else (int(groups["count"]), int(groups["keep"]))
        if not 1 <= self.top <= self.outputs or self.top > 32:
            raise ValueError(f"a token uses between 1 and min(experts, 32) experts, not {self.top} of {self.outputs}")
        if self.groups is not None:
            count, keep = self.groups
            if count < 1 or self.outputs % count or not 1 <= keep <= count or keep * (self.outputs // count) < self.top:
                raise ValueError("the experts form equal groups, and the kept groups hold enough of them")
        self.chosen_apart = bool(self.correction or self.groups or self.identities or self.weight_scale != 1.0)
        if self.chosen_apart and score == "chosen":
            raise ValueError("a correction, groups, identities and a weight factor go with sigmoid or softmax scores")
        if weight_on not in ("input", "output"):
            raise ValueError("weight_on is 'input' or 'output'")
        if score not in ("sigmoid", "softmax", "chosen") or expert_act not in ("silu", "clamped", "relu2"):
            raise ValueError("score is 'sigmoid', 'softmax' or 'chosen', expert_act 'silu', 'clamped' or 'relu2'")
        self.router_bias, self.shared_gate = bool(router_bias), bool(shared_gate)
        if self.router_bias and score == "sigmoid":
            raise ValueError("a router bias goes with softmax or chosen-logit scores")
        if self.shared_gate and shared is None:
            raise ValueError("a gate on the shared feed-forward needs one")
        self.score, self.expert_act, self.limit, self.alpha = score, expert_act, float(limit), float(alpha)
        self.shared = None if shared is None else make_part("feed_forward", shared)
        if self.shared is not None:
            self.kernel_libs = type(self).kernel_libs + tuple(getattr(self.shared, "kernel_libs", ()))
        self.names = {"router": "ffn_router.weight", "router_bias": "ffn_router.bias", "correction": "ffn_router.correction",
                      "shared_gate": "ffn_shared_gate.weight", "gate": "ffn_gate.{e}.weight", "up": "ffn_up.{e}.weight",
                      "down": "ffn_down.{e}.weight", **(names or {})}

    def params(self):
        nm, p = self.names, {self.names["router"]: ParamDecl((self.outputs, self.hidden), "vector", init="conv")}
        if self.router_bias:
            p[nm["router_bias"]] = ParamDecl((self.outputs,), "vector", init="conv")
        if self.correction:
            p[nm["correction"]] = ParamDecl((self.outputs,), "vector", init="conv")
        if self.shared_gate:
            p[nm["shared_gate"]] = ParamDecl((1, self.hidden), "vector", init="conv")
        for e in range(self.experts):
            if self.expert_act != "relu2":
                p[nm["gate"].format(e=e)] = ParamDecl((self.ff_dim, self.hidden))
            p[nm["up"].format(e=e)] = ParamDecl((self.ff_dim, self.hidden))
            p[nm["down"].format(e=e)] = ParamDecl((self.hidden, self.ff_dim))
        if self.shared is not None:
            p.update(self.shared.params())
        return p

    def bind(self, tensors, dtype):
        nm, E = self.names, range(self.experts)
        if self.shared is not None:
            self.shared.bind({k: tensors[k] for k in self.shared.params()}, dtype)
        self.w_router = tensors[nm["router"]].float()
        if self.shared_gate:                 # one more row of the router's product
            self.w_router = torch.cat([self.w_router, tensors[nm["shared_gate"]].float().reshape(1, self.hidden)], dim=0)
        self.w_router = self.w_router.contiguous()
        self.b_router = tensors[nm["router_bias"]].float().contiguous() if self.router_bias else None
        self.w_correction = tensors[nm["correction"]].float().contiguous() if self.correction else None
        if self.expert_act == "relu2":
            self.w_gate_up = torch.stack([tensors[nm["up"].format(e=e)] for e in E]).contiguous()  # [E, F, hidden]
        else:
            self.w_gate_up = torch.stack([torch.cat([tensors[nm["gate"].format(e=e)], tensors[nm["up"].format(e=e)]], dim=0)
                                          for e in E]).contiguous()                              # [E, 2F, hidden]
        self.w_down = torch.stack([tensors[nm["down"].format(e=e)] for e in E]).contiguous()   # [E, hidden, F]
        self.dtype = dtype

    def _routed(self, x, step, unit, onto=None):
        """The experts' sum with the shared feed-forward's rows in it."""
        more = {}
        if self.chosen_apart:
            more = dict(correction=self.w_correction, groups=self.groups, identities=self.identities, weight_scale=self.weight_scale)
        if onto is not None:
            more["onto"] = onto
        return step.ops.routed_experts(x, self.w_router, self.w_gate_up, self.w_down, self.top, self.renormalize, self.weight_on,
                                       score=self.score, act=self.expert_act, limit=self.limit, alpha=self.alpha,
                                       router_bias=self.b_router, unit=unit, unit_gated=self.shared_gate, **more)

    def forward(self, x, step):
        ops = step.ops
        if self.score == "chosen" or self.expert_act == "relu2" or self.router_bias or self.shared_gate or self.chosen_apart:
            # the shared feed-forward's rows join in the sum over the chosen experts
            return self._routed(x, step, None if self.shared is None else self.shared.forward(x, step))
        if self.score == "sigmoid" and self.expert_act == "silu":
            y = ops.routed_experts(x, self.w_router, self.w_gate_up, self.w_down, self.top, self.renormalize, self.weight_on)
        else:
            y = ops.routed_experts(x, self.w_router, self.w_gate_up, self.w_down, self.top, self.renormalize, self.weight_on,
                                   score=self.score, act=self.expert_act, limit=self.limit, alpha=self.alpha)
        if self.shared is None:
            return y
        return ops.weighted_sum(y, self.shared.forward(x, step), 1.0, 1.0)

    def forward_onto(self, x, step, h, other, cast=True):
        """The combine adds the experts' sum and `other` to the residual stream itself."""
        return self._routed(x, step, None if self.shared is None else self.shared.forward(x, step), onto=(h.data, other, cast))


register_part("feed_forward", "swiglu", SwiGlu)
register_part("feed_forward", "routed_experts", RoutedExperts)
register_part("feed_forward", "clamped_glu", ClampedGlu)
register_part("feed_forward", "dense", DenseMlp)
