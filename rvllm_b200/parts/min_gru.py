"""minGRU: a gated recurrence, channel by channel, whose gates read only the current token.

    z = sigmoid(Wz h + bz),   u = Wx h + bx,   c = u + 1/2 where u >= 0, sigmoid(u) where u < 0
    S_t = (1 - z) S_(t-1) + z c,  S starts at zero;    y = Wo (S_t * silu(Wg h))

(Feng et al., "Were RNNs All We Needed?".)  One stacked product gives [z | x | g] in float32.  A request keeps one float32
row of `width` channels, which the cache manager zeroes when the slot is handed out.  Gates, candidate and state are
float32; what enters the last product is rounded once.  Nothing is read on the host.
"""
from __future__ import annotations

import torch

from .base import MIXERS, Part, StateNeed, TensorSpec
from .linear import Linear


class MinGruMixer(Part):
    def __init__(self, hidden_size: int, width: int, names=("z", "x", "g", "o"), suffix: str = "", bias_suffix: str = ".b"):
        from ..errors import ConfigError
        if width < 1:
            raise ConfigError(f"a minGRU needs at least one channel, got {width}")
        self.hidden_size, self.width, self.names, self.bias_suffix = hidden_size, width, tuple(names), bias_suffix
        self.proj = Linear(hidden_size, [width, width, width], list(names[:3]), suffix=suffix)
        self.out = Linear(width, [hidden_size], [names[3]], suffix=suffix)
        self.z_bias = self.x_bias = None

    def tensor_specs(self):
        z, x = (n + self.bias_suffix for n in self.names[:2])
        return {**self.proj.tensor_specs(), **self.out.tensor_specs(),
                z: TensorSpec((self.width,), "bias"), x: TensorSpec((self.width,), "bias")}

    def bind(self, get):
        self.proj.bind(get)
        self.out.bind(get)
        self.z_bias, self.x_bias = (get(n + self.bias_suffix).float().contiguous() for n in self.names[:2])

    def cache_need(self):
        return StateNeed((self.width,), "float32")

    def __call__(self, x, ctx, cache, residual=None, write_cache=True, out_dtype=None):
        proj = self.proj(x, ctx, out_dtype=torch.float32)
        y = ctx.kernels.mingru(proj, self.z_bias, self.x_bias, ctx.cu_seqlens, ctx.state_slots, cache.state, self.width,
                               ctx.num_tokens == ctx.num_seqs, x.dtype)
        return self.out(y, ctx, residual=residual, out_dtype=out_dtype)


MIXERS.register("min_gru", MinGruMixer)
