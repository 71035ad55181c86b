"""State-space mixer with one decay per head (Mamba-2, state-space duality).

    [z | x | B | C | dt] = h . W_in^T                      z, x: heads x vdim;  B, C: groups x state;  dt: heads
    x, B, C <- silu(causal_conv(x, B, C) + conv bias)      one short depthwise convolution over time
    d = softplus(dt + dt_bias)                             a step size per head
    per head (head i uses group i // (heads / groups)):
        S <- exp(-exp(A_log) d) S + d B x^T;   y = S^T C + D x          S: state x vdim
    out = ( parts of (y * silu(z)) / rms(part) * norm weight ) . W_o^T  `norm_parts` equal parts of heads * vdim

Kept per request: S [heads, state, vdim] and the convolution's last taps - 1 inputs, both 32-bit, zero for a new request.
Step sizes, decays, the state, its sums, the gate and the norm are 32-bit in every mode; the projections and the
convolution's output follow the model's dtype.  `names` gives the tensors' names.
"""
from __future__ import annotations

from .base import Mixer, ParamDecl, StateNeed, register_part, stack_rows

DEFAULT_NAMES = {"in": "ssm_in.weight", "conv": "ssm_conv1d.weight", "conv_bias": "ssm_conv1d.bias", "dt_bias": "ssm_dt.bias",
                 "a_log": "ssm_a", "d": "ssm_d", "norm": "ssm_norm.weight", "o": "ssm_out.weight"}


class Mamba2(Mixer):
    accepts_lazy_input = True     # x goes straight into a product
    graph_safe = True             # forward launches kernels only; nothing is read back to the host
    kernel_libs = ("causal_conv", "mamba2")

    def __init__(self, hidden: int, heads: int, vdim: int, state: int, groups: int, taps: int, norm_parts: int, eps: float,
                 conv_bias: bool = True, names=None):
        self.hidden, self.heads, self.vdim, self.state = int(hidden), int(heads), int(vdim), int(state)
        self.groups, self.taps, self.norm_parts, self.eps = int(groups), int(taps), int(norm_parts), float(eps)
        self.conv_bias = bool(conv_bias)
        self.inner, self.channels = self.heads * self.vdim, self.heads * self.vdim + 2 * self.groups * self.state
        if self.heads % self.groups:
            raise ValueError(f"{self.heads} heads cannot share {self.groups} groups evenly")
        if self.inner % self.norm_parts:
            raise ValueError(f"{self.inner} values cannot be normed in {self.norm_parts} equal parts")
        if self.taps < 1 or self.taps > 16:
            raise ValueError(f"the convolution kernels take 1 to 16 taps, not {self.taps}")
        if not 1 <= self.state <= 512:
            raise ValueError(f"the recurrence's kernels take 1 to 512 states, not {self.state}")
        self.names = {**DEFAULT_NAMES, **(names or {})}

    def params(self):
        nm, I, C, H, L = self.names, self.inner, self.channels, self.heads, self.taps
        vec = lambda n, init="conv": ParamDecl((n,), "vector", init=init)
        p = {nm["in"]: ParamDecl((I + C + H, self.hidden)),
             nm["conv"]: ParamDecl((C, L), "vector", alt_shapes=((C, 1, L),), init="conv"),
             nm["dt_bias"]: vec(H), nm["a_log"]: vec(H), nm["d"]: vec(H, "norm_weight"), nm["norm"]: vec(I, "norm_weight"),
             nm["o"]: ParamDecl((self.hidden, I))}
        if self.conv_bias:
            p[nm["conv_bias"]] = vec(C)
        return p

    def cache_need(self):
        return (StateNeed((self.heads, self.state, self.vdim)), StateNeed((max(self.taps - 1, 1), self.channels)))

    def bind(self, tensors, dtype):
        nm, I, C = self.names, self.inner, self.channels
        w = tensors[nm["in"]]
        # z, x | B | C and dt each start on a 16-byte boundary of a row
        self.w_in, self.at = stack_rows([w[:I], w[I:I + C], w[I + C:]])
        self.conv_w = tensors[nm["conv"]].reshape(C, self.taps).float().contiguous()
        self.conv_b = tensors[nm["conv_bias"]].float().contiguous() if self.conv_bias else None
        self.dt_bias, self.a_log, self.d, self.norm_w = (tensors[nm[k]].float().contiguous() for k in ("dt_bias", "a_log", "d", "norm"))
        self.w_o = tensors[nm["o"]]
        self.dtype = dtype

    def forward(self, x, step, cache, write_cache=True):
        ops = step.ops
        matrix_state, conv_state = cache
        y = ops.linear(x, self.w_in)
        o = ops.mamba2(y, self.at, self.conv_w, self.conv_b, self.dt_bias, self.a_log, self.d, self.norm_w, self.eps, self.norm_parts,
                       matrix_state.state, conv_state.state, step, self.heads, self.groups, self.state, self.vdim, write_cache)
        return ops.linear(o, self.w_o)


register_part("mixer", "mamba2", Mamba2)
