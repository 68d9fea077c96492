"""The Sozudra design written out plainly: float64, whole sequences, no cache and no carried state, one function per
mechanism.

It shares nothing with the package: the tests compare the engine (its step function, cache, state rows, kernels) with
this.  Notation: h a sublayer's input [T, width]; u(v) = v / sqrt(mean(v^2) + eps) over the last dimension.

`store` is applied to every tensor that an engine keeps between two kernels (identity by default; `round_to_bfloat16`
measures what bfloat16 storage costs by itself, all arithmetic staying float64).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def _keep(t):
    return t


def round_to_bfloat16(t):
    return t.to(torch.bfloat16).to(torch.float64)


def unit_rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def embed(tokens: torch.Tensor, w, bigram: Optional[dict]) -> torch.Tensor:
    """A row per token plus a row per (previous token, token), found by a hash; the first token has the table's last row."""
    x = w["embed"][tokens]
    if bigram is None:
        return x
    rows = [bigram["buckets"]]
    for a, b in zip(tokens.tolist()[:-1], tokens.tolist()[1:]):
        rows.append((a * bigram["mul_prev"] + b * bigram["mul_cur"]) % bigram["buckets"])
    return x + w["bigram"][torch.tensor(rows)]


def pair_frequency(i: int, rot: dict) -> float:
    """Turn per position of pair i: base^(-2i/dims), and with a `scaling` that frequency and the one `factor` times lower
    blended by a ramp over the pair's number (YaRN)."""
    dims, base, s = rot["dims"], float(rot["base"]), rot.get("scaling")
    f = base ** (-2.0 * i / dims)
    if not s:
        return f

    def pair_turning(times: float) -> float:            # which pair turns `times` times over the original length
        return dims * math.log(s["original"] / (2.0 * math.pi * times)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_turning(s["fast"])), 0)
    hi = min(math.ceil(pair_turning(s["slow"])), dims - 1)
    ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
    return f / s["factor"] * ramp + f * (1.0 - ramp)


def turn_halves(v: torch.Tensor, positions: torch.Tensor, rot: dict) -> torch.Tensor:
    """v [T, ..., D]: the pairs (i, i + dims / 2) turn by position * frequency; the rest stays.  With a scaling the turned
    elements also grow by 0.1 ln(factor) + 1."""
    out = v.clone()
    half = rot["dims"] // 2
    grow = 0.1 * math.log(rot["scaling"]["factor"]) + 1.0 if rot.get("scaling") else 1.0
    shape = [v.shape[0]] + [1] * (v.dim() - 2)
    for i in range(half):
        ang = (positions.to(torch.float64) * pair_frequency(i, rot)).reshape(shape)
        c, s = grow * torch.cos(ang), grow * torch.sin(ang)
        a, b = v[..., i], v[..., i + half]
        out[..., i] = a * c - b * s
        out[..., i + half] = b * c + a * s
    return out


def visible_weights(q: torch.Tensor, k: torch.Tensor, positions, scale: float, cap: Optional[float], window: Optional[int]):
    """Softmax weights [T, T] of one head: capped scores, a query sees itself and the window - 1 positions before it."""
    score = (q @ k.T) * scale
    if cap is not None:
        score = cap * torch.tanh(score / cap)
    dist = positions[:, None] - positions[None, :]
    hidden = dist < 0
    if window is not None:
        hidden = hidden | (dist >= window)
    return torch.softmax(score.masked_fill(hidden, float("-inf")), -1)


def _window(m: dict) -> Optional[int]:
    return m["mask"]["size"] if m.get("mask") else None


def turned_value_attention(h, w, p: str, m: dict, eps: float, positions, store=_keep) -> torch.Tensor:
    """Grouped heads, queries and keys turned and then made unit-RMS; a value is turned by its own position, and what a
    query collects is turned back by the query's."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = store(unit_rms(turn_halves((h @ w[p + "q"].T).reshape(T, H, D), positions, m["rot"]), eps))
    k = store(unit_rms(turn_halves((h @ w[p + "k"].T).reshape(T, G, D), positions, m["rot"]), eps))
    value_rot = {"dims": V, "base": m["rot"]["base"]}
    v = store(turn_halves((h @ w[p + "v"].T).reshape(T, G, V), positions, value_rot))
    heads = []
    for i in range(H):
        g = i // (H // G)
        got = store(visible_weights(q[:, i], k[:, g], positions, m["scale"], m.get("softcap"), _window(m)) @ v[:, g])
        heads.append(store(turn_halves(got, -positions, value_rot)))
    return torch.cat(heads, dim=1) @ w[p + "o"].T


def min_gru(h, w, p: str, m: dict, store=_keep) -> torch.Tensor:
    """S <- (1 - z) S + z c, element by element, walked token by token from zero."""
    z = torch.sigmoid(h @ w[p + "z"].T + w[p + "z.b"])
    u = h @ w[p + "x"].T + w[p + "x.b"]
    c = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    g = h @ w[p + "g"].T
    S = torch.zeros(m["width"], dtype=h.dtype)
    out = torch.zeros_like(c)
    for t in range(h.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * c[t]
        out[t] = S
    return store(out * g * torch.sigmoid(g)) @ w[p + "o"].T


def side_by_side(h, w, p: str, m: dict, eps: float, positions, store=_keep) -> torch.Tensor:
    return m["left_scale"] * turned_value_attention(h, w, p + "left.", m["left"], eps, positions, store) \
        + m["right_scale"] * min_gru(h, w, p + "right.", m["right"], store)


def map_difference(w, p: str, diff: float) -> float:
    """The factor on the second map, one number for the layer."""
    return float(torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum())) + diff


def differential_attention(h, w, p: str, m: dict, eps: float, positions, store=_keep) -> torch.Tensor:
    """Two softmax maps per head over the same values, the second taken off the first; unit RMS per head."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, 2, D)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, 2, D)
    v = store((h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, V))
    q, k = store(turn_halves(q, positions, m["rot"])), store(turn_halves(k, positions, m["rot"]))
    lam = map_difference(w, p, m["diff"])
    heads = []
    for i in range(H):
        g = i // (H // G)
        a1, a2 = (store(visible_weights(q[:, i, j], k[:, g, j], positions, m["scale"], m.get("softcap"), _window(m)) @ v[:, g])
                  for j in (0, 1))
        heads.append(store(unit_rms(a1 - lam * a2, eps) * (1.0 - m["diff"])))
    return torch.cat(heads, dim=1) @ w[p + "o"].T


def gated_expert(h, w, p: str, store=_keep) -> torch.Tensor:
    a = h @ w[p + "gate"].T
    return store(a * torch.sigmoid(a) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p: str, router: dict):
    """The `top` experts with the largest logits (bias included), weighted by a softmax over those logits alone."""
    z = h @ w[p + "router"].T + w[p + "router.b"]
    best = z.topk(router["top"], dim=-1)
    return best.indices, torch.softmax(best.values, -1)


def moe(h, w, p: str, mlp: dict, store=_keep) -> torch.Tensor:
    chosen, weights = route(h, w, p, mlp["router"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, slots = torch.nonzero(chosen == e, as_tuple=True)
        if len(rows):
            out[rows] += weights[rows, slots][:, None] * gated_expert(h[rows], w, f"{p}e{e}.", store)
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * gated_expert(h, w, p + "shared.", store)
    return out


def layer_order(cfg: dict) -> List[int]:
    """Which layer runs when: the looped span's passes in a row, each layer number once per pass."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    span = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + span * loop["times"] + list(range(loop["stop"], n))


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], store=_keep, streams: Optional[list] = None) -> torch.Tensor:
    """float64 logits [T, vocab]; `streams` collects the residual stream after every layer run."""
    w = {k: (v.to(torch.float64) if v.is_floating_point() else v.long()) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    tok = torch.as_tensor(list(tokens), dtype=torch.long)
    pos = torch.arange(len(tok))
    x = embed(tok, w, (cfg.get("embedding") or {}).get("bigram"))
    for i in layer_order(cfg):
        layer = cfg["layers"][i]
        p, m = f"l{i}.", layer["mixer"]
        h = store(unit_rms(x, eps) * w[p + "norm1"])
        if layer["type"] == "parallel":
            y = side_by_side(h, w, p + "mix.", m, eps, pos, store)
        elif layer["type"] == "attention":
            y = differential_attention(h, w, p + "mix.", m, eps, pos, store)
        else:
            raise ValueError(layer["type"])
        if layer.get("mlp"):
            y = y + moe(store(unit_rms(x, eps) * w[p + "norm2"]), w, p + "mlp.", layer["mlp"], store)
        x = x + cfg["residual_mult"] * y
        if streams is not None:
            streams.append(x.clone())
    return store(unit_rms(x, eps) * w["final.norm"]) @ w["head"].T


def greedy(cfg: dict, weights, prompt: List[int], n: int) -> List[int]:
    toks, out = list(prompt), []
    for _ in range(n):
        nxt = int(torch.argmax(forward(cfg, weights, toks)[-1]))
        out.append(nxt)
        toks.append(nxt)
    return out
