"""The two ends of a model, the token embedding and the linear head, and what layers take from a token's row of another table.

The embedding gathers rows of its table into the 32-bit residual stream (the reference gathers on
the host, src/transformer/embedding.zig:6-31); the head multiplies the final norm's rows with its
matrix into 32-bit logits (src/main.zig:867-881).  When the embedding is tied the head uses the
embedding's table (src/loader/gguf_model.zig:47-54).
"""
from __future__ import annotations

import torch

from .base import Embedding, Head, NormedTerm, ParamDecl, Part, TokenInput, register_part


class TokenEmbedding(Embedding):
    graph_safe = True      # forward launches kernels only; nothing is read back to the host

    def __init__(self, weight: str, vocab: int, hidden: int, scale: float = 1.0, sinusoidal=None):
        """`sinusoidal=base`: a vector of the token's position is added to its row, sines in the even and cosines in the odd
        entries, entries 2i and 2i + 1 turning by base^(-2i/hidden) a position."""
        self.weight_name, self.vocab, self.hidden = weight, int(vocab), int(hidden)
        self.scale = float(scale)          # the gathered rows are multiplied by it (in 32-bit)
        self.sinusoidal = None if sinusoidal is None else float(sinusoidal)
        if self.sinusoidal is not None and self.sinusoidal <= 0:
            raise ValueError("the base of the position vectors is positive")
        self.table = None

    def params(self):
        return {self.weight_name: ParamDecl((self.vocab, self.hidden), "table")}

    def bind(self, tensors, dtype):
        self.table = tensors[self.weight_name]

    def forward(self, token_ids, step):
        if self.sinusoidal is not None:
            return step.ops.embed(token_ids, self.table, self.scale, step.positions, self.sinusoidal)
        if self.scale != 1.0:
            return step.ops.embed(token_ids, self.table, self.scale)
        return step.ops.embed(token_ids, self.table)


class LinearHead(Head):
    accepts_lazy_input = True     # x goes straight into a product
    graph_safe = True

    def __init__(self, weight: str, tied: bool, vocab: int, hidden: int, scale: float = 1.0, softcap=None):
        self.weight_name, self.tied, self.vocab, self.hidden = weight, bool(tied), int(vocab), int(hidden)
        self.scale = float(scale)                                   # logits = product * scale ...
        self.softcap = None if not softcap else float(softcap)      # ... then cap * tanh(logits / cap), in 32-bit
        self.w = None

    def params(self):
        return {} if self.tied else {self.weight_name: ParamDecl((self.vocab, self.hidden), "matrix")}

    def bind(self, tensors, dtype):
        if not self.tied:
            self.w = tensors[self.weight_name]

    def tie(self, embedding):
        self.w = embedding.table

    def forward(self, x, step):
        logits = step.ops.linear(x, self.w, out_dtype=torch.float32)
        if self.scale != 1.0 or self.softcap is not None:
            logits = step.ops.scale_softcap(logits, self.scale, self.softcap)
        return logits


class TokenTable(Part):
    """A table by token id that layers read by themselves: [vocab, columns] in the model's dtype.  What a layer takes from a
    token's row is the layer's business."""
    graph_safe = True

    def __init__(self, weight: str, columns: int, vocab: int):
        self.weight_name, self.vocab, self.columns = weight, int(vocab), int(columns)
        self.table = None

    def params(self):
        return {self.weight_name: ParamDecl((self.vocab, self.columns), "table")}

    def bind(self, tensors, dtype):
        self.table = tensors[self.weight_name].to(dtype)


class TokenSideInput(TokenInput):
    """A layer's term from its part of the token's row in a table (columns `at` .. `at + dim - 1` of the table named `table`):

        g = gelu_tanh(gate x) * row[at : at + dim];   y = proj g;   h = h + y / sqrt(mean(y^2) + eps) * norm

    The lookup is part of the gate product's epilogue (few rows) or of the activation behind it; the norm and the addition
    belong to the next norm's kernel.  `names`: gate, proj, norm."""
    graph_safe = True

    def __init__(self, hidden: int, dim: int, at: int, eps: float, table: str, names=None):
        self.hidden, self.dim, self.at, self.eps, self.table_name = int(hidden), int(dim), int(at), float(eps), table
        self.names = {"gate": "token_gate.weight", "proj": "token_proj.weight", "norm": "token_norm.weight", **(names or {})}
        self.table = None

    def params(self):
        return {self.names["gate"]: ParamDecl((self.dim, self.hidden)), self.names["proj"]: ParamDecl((self.hidden, self.dim)),
                self.names["norm"]: ParamDecl((self.hidden,), "vector", init="norm_weight")}

    def bind(self, tensors, dtype):
        self.w_gate, self.w_proj, self.w_norm = (tensors[self.names[k]] for k in ("gate", "proj", "norm"))

    def attach(self, tables):
        self.table = tables[self.table_name].table

    def forward(self, x, step):
        g = step.ops.linear_side(x, self.w_gate, self.table, step.token_ids, self.at)
        return NormedTerm(step.ops.linear(g, self.w_proj), self.w_norm, self.eps)


register_part("table", "token_table", TokenTable)
register_part("token_input", "side_rows", TokenSideInput)
register_part("embedding", "embedding", TokenEmbedding)
register_part("head", "linear_head", LinearHead)
