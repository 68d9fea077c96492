"""Differential attention: two softmax maps per head over the same values, one taken off the other, over the paged cache.

    q = Wq h + bq  (per head two maps of `head_dim`: [map 1 | map 2]),  k = Wk h + bk likewise per kv head,  v = Wv h + bv
    the leading rotary elements of every map of every head of q and k are turned by the position
    s_m = scale * (q_m . k_m), with a cap s_m <- cap tanh(s_m / cap);  i sees j with 0 <= i - j < window;  a_m = softmax(s_m) v
    lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff                              one number for the layer
    o = a_1 - lambda a_2;   o <- (1 - diff) o / sqrt(mean(o^2) + eps) per head;   y = Wo [o_1 .. o_H]

(Ye et al., "Differential Transformer".)  Each token caches ONE row per kv head, [k_1 | k_2], and one value, read by both maps: a
query row of map 1 is [q_1 | 0] and one of map 2 is [0 | q_2], so that its product with the key row is that map's score, and
the attention kernels of the engine serve 2 H heads on G kv heads as they are.  (The zeros cost one product of `head_dim`
per score; caching two pairs of heads instead would cost a second copy of every value.)  A head's slot is
max(2 head_dim, value_dim) wide, rounded up to a multiple of 16, the rest zeros.  One stacked product gives [q | k | v] in
float32; one kernel adds the biases, rotates and writes the cache; one kernel forms the difference, its norm and factor.
lambda is formed once, in double precision, when the tensors are bound.
"""
from __future__ import annotations

from typing import Optional

import torch

from .base import MIXERS, KvCacheNeed, Part, TensorSpec
from .linear import Linear


class DifferentialAttention(Part):
    LAMBDAS = ("lq1", "lk1", "lq2", "lk2")
    SLOT_MULTIPLE = 16
    PAIRS = ("neighbours", "halves")

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, value_dim: int, scale: float, diff: float,
                 eps: float, softcap: Optional[float] = None, window: Optional[int] = None, bias: bool = True,
                 pairs: str = "halves", position=None, suffix: str = "", bias_suffix: str = ".b"):
        from ..errors import ConfigError
        problems = []
        if min(num_heads, num_kv_heads, head_dim, value_dim) < 1 or num_heads % max(num_kv_heads, 1):
            problems.append(f"{num_heads} query heads of 2 x {head_dim} on {num_kv_heads} key/value heads of 2 x {head_dim} / {value_dim}")
        self.slot_dim = -(-max(2 * head_dim, value_dim) // self.SLOT_MULTIPLE) * self.SLOT_MULTIPLE
        if self.slot_dim > 1024:
            problems.append(f"a head's two maps and its value have at most 1,024 elements, got 2 x {head_dim} and {value_dim}")
        if softcap is not None and not softcap > 0:
            problems.append(f"the score cap must be positive, got {softcap}")
        if window is not None and window < 1:
            problems.append(f"the window must span at least one key, got {window}")
        if pairs not in self.PAIRS:
            problems.append(f"rotation pairs {pairs!r} are not known ({', '.join(self.PAIRS)})")
        if problems:
            raise ConfigError(problems, "differential attention")
        self.hidden_size, self.num_heads, self.num_kv_heads = hidden_size, num_heads, num_kv_heads
        self.head_dim, self.value_dim, self.scale, self.diff, self.eps = head_dim, value_dim, scale, float(diff), eps
        self.softcap, self.window, self.pairs, self.position = softcap, window, pairs, position
        self.proj = Linear(hidden_size, [2 * num_heads * head_dim, 2 * num_kv_heads * head_dim, num_kv_heads * value_dim],
                           ["q", "k", "v"], bias=bias, suffix=suffix, bias_suffix=bias_suffix)
        self.out = Linear(num_heads * value_dim, [hidden_size], ["o"], suffix=suffix)
        self.bias = None
        self.lam: Optional[float] = None

    def tensor_specs(self):
        return {**self.proj.tensor_specs(), **self.out.tensor_specs(),
                **{n: TensorSpec((self.head_dim,), "mixing") for n in self.LAMBDAS}}

    def bind(self, get):
        self.proj.bind(get)
        self.out.bind(get)
        self.bias = self.proj.bias.float().contiguous() if self.proj.bias is not None else None    # added to float32 rows
        q1, k1, q2, k2 = (get(n).double() for n in self.LAMBDAS)
        self.lam = float(torch.exp((q1 * k1).sum()) - torch.exp((q2 * k2).sum())) + self.diff

    def cache_need(self):
        return KvCacheNeed(self.num_kv_heads, self.slot_dim, self.window)

    def __call__(self, x, ctx, cache, residual=None, write_cache=True, out_dtype=None):
        from ..errors import ConfigError
        if not write_cache:
            raise ConfigError("a differential attention layer writes its own keys and values")
        k = ctx.kernels
        meta = ctx.attention[cache.group]
        tables = self.position.rotation_tables() if self.position is not None else None
        cos, sin = tables if tables is not None else (None, None)
        proj = self.proj(x, ctx, out_dtype=torch.float32, with_bias=False)        # rounded once, after bias and rotation
        q, _ = k.qk_prepare(proj, ctx.positions, cos, sin, meta.slot_mapping, cache.kv, self.num_heads, self.num_kv_heads,
                            self.head_dim, self.value_dim, self.slot_dim, x.dtype, halves=self.pairs == "halves", maps=2, bias=self.bias)
        o = k.paged_attention(q, cache.kv, meta, 2 * self.num_heads, self.num_kv_heads, self.slot_dim, self.scale, self.window,
                              softcap=self.softcap)
        o = k.map_difference(o, self.lam, self.eps, 1.0 - self.diff, self.num_heads, self.value_dim, self.slot_dim)
        return self.out(o, ctx, residual=residual, out_dtype=out_dtype)


MIXERS.register("differential_attention", DifferentialAttention)
