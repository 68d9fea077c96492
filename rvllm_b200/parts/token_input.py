"""Inputs that depend on token ids alone: one added to the stream at the end of a layer, one to the embedded tokens.

    e = table[token][column : column + dim]        one table for all layers, each layer its own columns
    g = gelu_tanh(W_gate x) * e                    x: the stream itself (no norm in front)
    y = W_proj g;   x <- x + y / sqrt(mean(y^2) + eps) * w

`token_table_rows` is the hook that looks the step's tokens up in the table ONCE per step (tensor named in full, as
the checkpoint names it) and leaves the rows in `ctx.extras[key]`; `token_side_input` is the per-layer part, a
feed-forward by interface, that reads its columns of those rows.  The norm's weight is a plain one.

`bigram_rows` adds, to the embedded tokens, a row found by the pair (previous token, token):

    x <- x + table[ (previous * mul_prev + token * mul_cur) mod buckets ]          float32; the start of a float32 stream

and the table's last row, number `buckets`, for a sequence's first token.  The previous token is part of a sequence's
state: an int32 state row that the step leaves the sequence's last token in.
"""
from __future__ import annotations

import torch

from .base import FEED_FORWARDS, HOOKS, Part, StateNeed, TensorSpec
from .linear import Linear


class TokenTableRows(Part):
    names_in_full = True

    def __init__(self, rows: int, width: int, tensor: str, key: str):
        self.rows, self.width, self.tensor, self.key = rows, width, tensor, key
        self.table = None

    def tensor_specs(self):
        return {self.tensor: TensorSpec((self.rows, self.width), "matrix")}

    def bind(self, get):
        self.table = get(self.tensor)

    def __call__(self, x, ctx):
        ctx.extras[self.key] = ctx.kernels.gather_rows(self.table, ctx.token_ids)
        return x


class TokenSideInput(Part):
    def __init__(self, hidden_size: int, dim: int, column: int, eps: float, table: str):
        self.hidden_size, self.dim, self.column, self.eps, self.table = hidden_size, dim, column, eps, table
        self.gate = Linear(hidden_size, [dim], ["gate"], suffix="")
        self.proj = Linear(dim, [hidden_size], ["proj"], suffix="")
        self.norm = None

    def tensor_specs(self):
        return {**self.gate.tensor_specs(), **self.proj.tensor_specs(), "norm": TensorSpec((self.hidden_size,), "norm")}

    def bind(self, get):
        self.gate.bind(get)
        self.proj.bind(get)
        self.norm = get("norm")

    def __call__(self, x, ctx, residual=None, out_dtype=None):
        """x: the stream in the activations' type; residual: the float32 stream, updated in place."""
        k = ctx.kernels
        g = self.gate(x, ctx, out_dtype=torch.float32)
        g = k.gelu_mul_columns(g, ctx.extras[self.table], self.column, x.dtype)
        y = self.proj(g, ctx, out_dtype=torch.float32)
        return k.residual_rmsnorm(y, self.norm, self.eps, residual, None)[0]


class BigramRows(Part):
    names_in_full = True

    def __init__(self, width: int, buckets: int, mul_prev: int, mul_cur: int, tensor: str):
        from ..errors import ConfigError
        if buckets < 1:
            raise ConfigError(f"a bigram table needs at least one bucket, got {buckets}")
        self.width, self.buckets, self.mul_prev, self.mul_cur, self.tensor = width, buckets, mul_prev, mul_cur, tensor
        self.table = None

    def tensor_specs(self):
        return {self.tensor: TensorSpec((self.buckets + 1, self.width), "matrix")}

    def bind(self, get):
        self.table = get(self.tensor)

    def cache_need(self):
        return StateNeed((1,), "int32")

    def __call__(self, x, ctx, cache):
        return ctx.kernels.bigram_add(x, self.table, ctx.token_ids, ctx.positions, ctx.token_seq, ctx.cu_seqlens, ctx.state_slots,
                                      cache.state, self.mul_prev, self.mul_cur, self.buckets)


HOOKS.register("bigram_rows", BigramRows)
HOOKS.register("token_table_rows", TokenTableRows)
FEED_FORWARDS.register("token_side_input", TokenSideInput)
