"""Grouped-query attention with RMSNorms on the queries and keys of a head, and what may go with them: biases, a rotation behind
the norm or no positions at all but a learned bias per distance, a temperature on the query, capped scores, a window, a sink of
score zero, values mixed with those of an earlier layer, a gate per element of the result.

    q = Wq h + bq, k = Wk h + bk  (per head `head_dim`),  v = Wv h + bv  (per kv head `value_dim`)
    q <- q / sqrt(mean(q^2) + eps) * wq,  k likewise with wk            per head, one weight for all heads
    the leading rotary elements of every head of q and k are turned     (option `position`), pairs (2i, 2i + 1) or (i, i + half)
    q <- q (1 + c ln(floor((p + 1) / every) + 1)) at position p         (option `temperature` = (c, every))
    v <- (1 - l) v + l v_first                                           (option `value_mix`, below)
    s = scale * (q . k), with a cap s <- cap tanh(s / cap), plus a bias of (distance, head)   (option `distance_limit`; parts/distance.py)
    keys j with 0 <= i - j < window (no window: j <= i);  softmax, with `unit_sink` one more exp(0) in the denominator
    o <- o * sigmoid(Wg h)  element by element over all heads            (option `gate`)
    y = Wo [o_1 .. o_H]

`value_mix`: "first" leaves this layer's values (before anything else happens to them) in the step's `ctx.extras`; "later" takes a
share l (tensor `vmix`, one number) of those of the same token.  What is cached is the mixed value, so that only the layers of
one step exchange anything.  A layer with "first" has the tensor too, and does not use it.

A head's slot in the cache and in the attention kernels is `max(head_dim, value_dim)` wide, rounded up to a multiple of 16, the
shorter of key and value followed by zeros.  One stacked product gives [q | k | v | gate logits] in float32; one kernel adds the
biases, norms, turns, mixes and writes the cache; the kernel that gates the result also drops the slot's zeros (without a gate
the output matrix gets zero columns for them).  Sizes and constants are parameters; tensors: q, k, v (with biases), q.norm,
k.norm, vmix, rel, g, o.
"""
from __future__ import annotations

from typing import Optional, Tuple

import torch

from .base import MIXERS, KvCacheNeed, Part, TensorSpec
from .distance import distance_table
from .linear import Linear


class NormedQkAttention(Part):
    PAIRS = ("neighbours", "halves")
    VALUE_MIX = (None, "first", "later")
    SLOT_MULTIPLE = 16
    KEY = "first_values"

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, value_dim: int, scale: float, eps: float,
                 bias: bool = True, position=None, pairs: str = "neighbours", softcap: Optional[float] = None,
                 window: Optional[int] = None, distance_limit: Optional[float] = None, distance_rows: int = 32,
                 unit_sink: bool = False, temperature: Optional[Tuple[float, int]] = None, value_mix: Optional[str] = None,
                 gate: bool = False, suffix: str = "", bias_suffix: str = ".b"):
        from ..errors import ConfigError
        problems = []
        if min(num_heads, num_kv_heads, head_dim, value_dim) < 1 or num_heads % max(num_kv_heads, 1):
            problems.append(f"{num_heads} query heads of {head_dim} on {num_kv_heads} key/value heads of {head_dim} / {value_dim}")
        self.slot_dim = -(-max(head_dim, value_dim) // self.SLOT_MULTIPLE) * self.SLOT_MULTIPLE
        if self.slot_dim > 1024:
            problems.append(f"key and value sizes are at most 1,024, got {head_dim} and {value_dim}")
        if pairs not in self.PAIRS:
            problems.append(f"rotation pairs {pairs!r} are not known ({', '.join(self.PAIRS)})")
        if softcap is not None and not softcap > 0:
            problems.append(f"the score cap must be positive, got {softcap}")
        if window is not None and window < 1:
            problems.append(f"the window must span at least one key, got {window}")
        if temperature is not None and temperature[1] < 1:
            problems.append(f"the query temperature grows every {temperature[1]} positions; it must be at least 1")
        if value_mix not in self.VALUE_MIX:
            problems.append(f"value mixing {value_mix!r} is not known (first, later)")
        if problems:
            raise ConfigError(problems, "attention with normed queries and keys")
        self.hidden_size, self.num_heads, self.num_kv_heads = hidden_size, num_heads, num_kv_heads
        self.head_dim, self.value_dim, self.scale, self.eps = head_dim, value_dim, scale, eps
        self.position, self.pairs, self.softcap, self.window = position, pairs, softcap, window
        self.distance_limit, self.distance_rows, self.unit_sink = distance_limit, distance_rows, unit_sink
        self.temperature, self.value_mix, self.has_gate = temperature, value_mix, gate
        outs, names = [num_heads * head_dim, num_kv_heads * head_dim, num_kv_heads * value_dim], ["q", "k", "v"]
        self.qkv_columns = sum(outs)
        # (the gate's matrix has no bias: it is stacked behind the others when the tensors are bound)
        self.qkv = Linear(hidden_size, outs, names, bias=bias, suffix=suffix, bias_suffix=bias_suffix)
        self.gate = Linear(hidden_size, [num_heads * value_dim], ["g"], suffix=suffix) if gate else None
        self.out = Linear(num_heads * value_dim, [hidden_size], ["o"], suffix=suffix)
        self.q_norm = self.k_norm = self.bias = self.weight = self.distance_bias = self.sinks = None
        self.lam: Optional[float] = None

    def tensor_specs(self):
        specs = {**self.qkv.tensor_specs(), **self.out.tensor_specs(),
                 "q.norm": TensorSpec((self.head_dim,), "norm"), "k.norm": TensorSpec((self.head_dim,), "norm")}
        if self.gate is not None:
            specs.update(self.gate.tensor_specs())
        if self.distance_limit is not None:
            specs["rel"] = TensorSpec((self.distance_rows, self.num_heads), "mixing", free=(0,))
        if self.value_mix is not None:
            specs["vmix"] = TensorSpec((), "coef")
        return specs

    def bind(self, get):
        self.qkv.bind(get)
        self.out.bind(get)
        self.weight = self.qkv.weight
        if self.gate is not None:
            self.gate.bind(get)
            self.weight = torch.cat([self.qkv.weight, self.gate.weight.to(self.qkv.weight.dtype)], dim=0).contiguous()
            self.gate.weight = None
        self.qkv.weight = None
        self.bias = self.qkv.bias.float().contiguous() if self.qkv.bias is not None else None      # added to float32 rows
        self.q_norm, self.k_norm = get("q.norm").float().contiguous(), get("k.norm").float().contiguous()
        if self.distance_limit is not None:
            self.distance_bias = distance_table(get("rel"), self.distance_limit, self.num_kv_heads)
        if self.unit_sink:
            self.sinks = torch.zeros((self.num_heads,), dtype=torch.float32, device=self.weight.device)
        if self.value_mix is not None:
            self.lam = float(get("vmix"))
        if self.slot_dim != self.value_dim and self.gate is None:          # zero columns where a head's slot is wider than its value
            w = self.out.weight.view(self.hidden_size, self.num_heads, self.value_dim)
            wide = torch.zeros((self.hidden_size, self.num_heads, self.slot_dim), dtype=w.dtype, device=w.device)
            wide[:, :, :self.value_dim] = w
            self.out.weight = wide.view(self.hidden_size, self.num_heads * self.slot_dim).contiguous()

    def cache_need(self):
        return KvCacheNeed(self.num_kv_heads, self.slot_dim, self.window)

    def __call__(self, x, ctx, cache, residual=None, write_cache=True, out_dtype=None):
        from ..errors import ConfigError
        if not write_cache:
            raise ConfigError("an attention layer with normed queries and keys writes its own keys and values")
        k = ctx.kernels
        meta = ctx.attention[cache.group]
        tables = self.position.rotation_tables() if self.position is not None else None
        cos, sin = tables if tables is not None else (None, None)
        T = x.shape[0]
        kept = first = None
        if self.value_mix == "first":
            kept = ctx.extras[self.KEY] = torch.empty((T, self.num_kv_heads * self.value_dim), dtype=torch.float32, device=x.device)
        elif self.value_mix == "later":
            first = ctx.extras[self.KEY]
        proj = k.linear(x, self.weight, None, None, torch.float32)        # rounded once, after bias, norm, rotation and mixing
        q, _ = k.qk_prepare(proj[:, :self.qkv_columns] if self.gate is not None else proj, ctx.positions, cos, sin, meta.slot_mapping,
                            cache.kv, self.num_heads, self.num_kv_heads, self.head_dim, self.value_dim, self.slot_dim, x.dtype,
                            eps=self.eps, halves=self.pairs == "halves", bias=self.bias, norms=(self.q_norm, self.k_norm),
                            temperature=self.temperature, keep_values=kept, mix_values=None if first is None else (first, self.lam))
        o = k.paged_attention(q, cache.kv, meta, self.num_heads, self.num_kv_heads, self.slot_dim, self.scale, self.window,
                              softcap=self.softcap, sinks=self.sinks, distance_bias=self.distance_bias)
        if self.gate is not None:
            o = k.gate_elements(o, proj, self.qkv_columns, self.num_heads, self.value_dim, self.slot_dim)
        return self.out(o, ctx, residual=residual, out_dtype=out_dtype)


MIXERS.register("normed_qk_attention", NormedQkAttention)
