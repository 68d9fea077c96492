"""The Lefolorn design written out plainly: float64, whole sequences, no cache and no carried state, one function per
mechanism.

It shares nothing with the package: the tests compare the engine (its step function, cache, kernels) with this.  Notation:
h a sublayer's input [T, width]; u(v) = v / sqrt(mean(v^2) + eps) over the last dimension.

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


def grouped_norm(x: torch.Tensor, w: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """Every one of `groups` equal consecutive parts over its own root mean square, then the weight."""
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    return unit_rms(parts, eps).reshape(x.shape) * w


def turn_neighbours(v: torch.Tensor, positions: torch.Tensor, rot: dict) -> torch.Tensor:
    """v [T, ..., D]: the pairs (2i, 2i + 1) of the leading `dims` elements turn by position * base^(-2i/dims)."""
    out = v.clone()
    shape = [v.shape[0]] + [1] * (v.dim() - 2)
    for i in range(rot["dims"] // 2):
        ang = (positions.to(torch.float64) * float(rot["base"]) ** (-2.0 * i / rot["dims"])).reshape(shape)
        c, s = torch.cos(ang), torch.sin(ang)
        a, b = v[..., 2 * i], v[..., 2 * i + 1]
        out[..., 2 * i] = a * c - b * s
        out[..., 2 * i + 1] = b * c + a * s
    return out


def distance_bucket(n: int, rows: int, limit: float) -> int:
    """Which row of a distance table of `rows` rows a key n positions back reads: the first half of the rows one distance
    each, the rest logarithmically up to `limit`, everything farther the last one."""
    near = rows // 2
    if n < near:
        return n
    return min(rows - 1, near + math.floor(math.log(n / near) / math.log(limit / near) * (rows - near)))


def query_temperature(positions: torch.Tensor, temp: Optional[dict]) -> torch.Tensor:
    """What a query at a position is multiplied by: it grows with the logarithm of the number of whole spans behind it."""
    if not temp:
        return torch.ones(len(positions), dtype=torch.float64)
    return torch.tensor([1.0 + temp["coef"] * math.log(math.floor((p + 1) / temp["every"]) + 1) for p in positions.tolist()],
                        dtype=torch.float64)


def head_weights(q, k, positions, scale: float, cap: Optional[float] = None, window: Optional[int] = None, table=None,
                 limit: float = 0.0, sink: Optional[float] = None) -> torch.Tensor:
    """Softmax weights [T, T] of one head.  `table` [rows]: added to a score by its distance's bucket; `sink`: a score without
    a value in the denominator (0 adds one to it)."""
    score = (q @ k.T) * scale
    if cap is not None:
        score = cap * torch.tanh(score / cap)
    dist = positions[:, None] - positions[None, :]
    if table is not None:
        T = len(positions)
        rows = torch.tensor([distance_bucket(n, len(table), limit) for n in range(T)])
        score = score + table[rows[dist.clamp(min=0)]]
    hidden = dist < 0
    if window is not None:
        hidden = hidden | (dist >= window)
    score = score.masked_fill(hidden, float("-inf"))
    if sink is None:
        return torch.softmax(score, -1)
    most = torch.clamp(score.max(-1, keepdim=True).values, min=float(sink))
    e = torch.exp(score - most)
    return e / (torch.exp(sink - most) + e.sum(-1, keepdim=True))


def projected_heads(h, w, p: str, m: dict, eps: float):
    """q [T, H, dim] and k [T, G, dim] under their norms, v [T, G, vdim]; all with biases."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, D), eps) * w[p + "q.norm"]
    k = unit_rms((h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, D), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, V)
    return q, k, v


def mix_values(v, w, p: str, m: dict, memory: dict):
    """The first layer that mixes values leaves its own behind; every later one takes a share `vmix` of those."""
    if not m.get("v_mix"):
        return v
    if "first" not in memory:
        memory["first"] = v
        return v
    lam = w[p + "vmix"]
    return (1.0 - lam) * v + lam * memory["first"].reshape(v.shape)


def biased_attention(h, w, p: str, m: dict, eps: float, positions, memory: dict, store=_keep) -> torch.Tensor:
    """No rotation: a learned number per (distance bucket, head), a temperature on the query, one in the denominator, an
    element-wise gate on the heads' results."""
    H, G = m["heads"], m["kv_heads"]
    q, k, v = projected_heads(h, w, p, m, eps)
    q = store(q * query_temperature(positions, m.get("q_temp"))[:, None, None])
    k, v = store(k), store(mix_values(v, w, p, m, memory))
    heads = []
    for i in range(H):
        g = i // (H // G)
        heads.append(store(head_weights(q[:, i], k[:, g], positions, m["scale"], table=w[p + "rel"][:, i], limit=m["bias_max"],
                                        sink=0.0) @ v[:, g]))
    return store(torch.cat(heads, dim=1) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def window_attention(h, w, p: str, m: dict, eps: float, positions, memory: dict, store=_keep) -> torch.Tensor:
    """Normed, then turned queries and keys; capped scores inside a window."""
    H, G = m["heads"], m["kv_heads"]
    q, k, v = projected_heads(h, w, p, m, eps)
    q, k = store(turn_neighbours(q, positions, m["rot"])), store(turn_neighbours(k, positions, m["rot"]))
    v = store(mix_values(v, w, p, m, memory))
    window = m["mask"]["size"] if m.get("mask") else None
    heads = []
    for i in range(H):
        g = i // (H // G)
        heads.append(store(head_weights(q[:, i], k[:, g], positions, m["scale"], cap=m.get("softcap"), window=window) @ v[:, g]))
    return torch.cat(heads, dim=1) @ w[p + "o"].T


def latent_attention(h, w, p: str, m: dict, eps: float, positions, store=_keep) -> torch.Tensor:
    """Queries through one low-rank row, keys and values of all heads through another; a sink per head."""
    T = h.shape[0]
    H, D, R, V, K = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = store(unit_rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"])
    q = (cq @ w[p + "uq"].T).reshape(T, H, D + R)
    q_rot = store(turn_neighbours(q[..., D:], positions, m["rot"]))
    down = h @ w[p + "dkv"].T
    c = store(unit_rms(down[:, :K], eps) * w[p + "dkv.norm"])
    r = store(turn_neighbours(down[:, K:], positions, m["rot"]))
    keys = (c @ w[p + "uk"].T).reshape(T, H, D)
    values = (c @ w[p + "uv"].T).reshape(T, H, V)
    heads = []
    for i in range(H):
        qq, kk = torch.cat([store(q[:, i, :D]), q_rot[:, i]], -1), torch.cat([keys[:, i], r], -1)
        heads.append(store(head_weights(qq, kk, positions, m["scale"], sink=float(w[p + "sink"][i])) @ values[:, i]))
    return torch.cat(heads, dim=1) @ w[p + "o"].T


def gated_expert(h, w, p: str, store=_keep) -> torch.Tensor:
    a = h @ w[p + "gate"].T
    return store(a * torch.sigmoid(a) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p: str, router: dict):
    """Softmax scores over experts and identity experts; chosen by score + correction inside the groups whose largest such sum
    is largest; weights: the chosen scores over their sum."""
    s = torch.softmax(h @ w[p + "router"].T, -1)
    c = s + w[p + "correction"]
    groups = router.get("groups") or {"count": 1, "keep": 1}
    best = c.reshape(h.shape[0], groups["count"], -1).max(-1).values.topk(groups["keep"], dim=-1).indices
    closed = torch.ones(h.shape[0], groups["count"], dtype=torch.bool).scatter_(1, best, False)
    c = c.masked_fill(closed.repeat_interleave(c.shape[1] // groups["count"], dim=1), float("-inf"))
    chosen = c.topk(router["top"], dim=-1).indices
    weights = s.gather(1, chosen)
    return chosen, weights / (weights.sum(-1, keepdim=True) + 1e-20)


def moe(h, w, p: str, mlp: dict, store=_keep) -> torch.Tensor:
    """An identity expert (the last ones of the router's outputs) gives back its input."""
    chosen, weights = route(h, w, p, mlp["router"])
    n = mlp["router"]["experts"]
    out = torch.zeros_like(h)
    for e in range(n + (mlp["router"].get("identity") or 0)):
        rows, slots = torch.nonzero(chosen == e, as_tuple=True)
        if len(rows):
            y = gated_expert(h[rows], w, f"{p}e{e}.", store) if e < n else h[rows]
            out[rows] += weights[rows, slots][:, None] * y
    if mlp.get("shared"):
        out = out + gated_expert(h, w, p + "shared.", store)
    return out


def sublayer_gate(h, w, p: str, n: int, store=_keep) -> torch.Tensor:
    """What sublayer n's result is multiplied by: a learned number per element times a sigmoid of the shared input."""
    return w[f"{p}ls{n}"] * torch.sigmoid(store(h @ w[f"{p}rg{n}"].T) + w[f"{p}rg{n}.b"])


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], store=_keep, streams: Optional[list] = None) -> torch.Tensor:
    """float64 logits [T, vocab]; `streams` collects the residual stream after every layer."""
    w = {k: (v.to(torch.float64) if v.is_floating_point() else v.long()) for k, v in weights.items()}
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    tok = torch.as_tensor(list(tokens), dtype=torch.long)
    pos = torch.arange(len(tok))
    x = w["embed"][tok]
    memory: dict = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = store(grouped_norm(x, w[p + "norm1"], groups, eps))
        if layer["type"] == "attention":
            y = biased_attention(h, w, p + "mix.", m, eps, pos, memory, store)
        elif layer["type"] == "attention_2":
            y = window_attention(h, w, p + "mix.", m, eps, pos, memory, store)
        elif layer["type"] == "latent_attention":
            y = latent_attention(h, w, p + "mix.", m, eps, pos, store)
        else:
            raise ValueError(layer["type"])
        y = y * sublayer_gate(h, w, p, 1, store)
        if layer.get("mlp"):
            y = y + moe(h, w, p + "mlp.", layer["mlp"], store) * sublayer_gate(h, w, p, 2, store)
        x = x + y
        if streams is not None:
            streams.append(x.clone())
    return store(grouped_norm(x, w["final.norm"], groups, eps)) @ w["head"].T


def greedy(cfg: dict, weights, prompt: List[int], n: int) -> List[int]:
    toks, out = list(prompt), []
    for _ in range(n):
        nxt = int(torch.argmax(forward(cfg, weights, toks)[-1]))
        out.append(nxt)
        toks.append(nxt)
    return out
