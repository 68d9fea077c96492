"""A learned bias per (distance between query and key, head), read from a table with fewer rows than distances.

The first half of the table's rows belong to one distance each; the others divide the distances up to `limit` logarithmically,
and everything farther reads the last row.  With R rows, N = R div 2, L = limit:

    row(n) = n  for n < N,  else  min(R - 1, N + floor( ln(n / N) / ln(L / N) * (R - N) ))

The attention kernels do not look rows up: `distance_table` writes the bias out per distance, up to the first distance from
which on the last row holds (a few hundred numbers per head), ordered so that the query heads of one key/value head lie side by
side - [kv heads, distances, heads per kv head] - and the rows of an attention tile, which are (token, head) pairs, read
neighbouring numbers.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import List

import torch

from ..errors import ConfigError

MAX_DISTANCES = 1 << 20


def bucket_rows(rows: int, limit: float) -> List[int]:
    """row(n) for n = 0, 1, ... up to the first n from which on the last row is read (that n included)."""
    near = rows // 2
    if rows < 2 or not limit > near:
        raise ConfigError(f"a distance table of {rows} rows needs a limit above {max(near, 1)}, got {limit}")
    out = list(range(near))
    while not out or out[-1] != rows - 1:
        n = len(out)
        if n > MAX_DISTANCES:
            raise ConfigError(f"a distance table that reaches beyond {MAX_DISTANCES} positions is not supported")
        out.append(min(rows - 1, near + math.floor(math.log(n / near) / math.log(limit / near) * (rows - near))))
    return out


@dataclass(frozen=True)
class DistanceBias:
    """`natural` and `log2` (the same times log2(e), for kernels that work in powers of two): float32
    [kv heads, distances, heads per kv head]; a distance beyond the last reads the last."""
    natural: torch.Tensor
    log2: torch.Tensor

    @property
    def distances(self) -> int:
        return self.natural.shape[1]

    @property
    def heads(self) -> int:
        return self.natural.shape[0] * self.natural.shape[2]


def distance_table(table: torch.Tensor, limit: float, num_kv_heads: int) -> DistanceBias:
    """`table` [rows, heads] as the checkpoint has it."""
    rows, heads = table.shape
    index = torch.tensor(bucket_rows(rows, limit), dtype=torch.long, device=table.device)
    by_distance = table.to(torch.float64)[index].view(len(index), num_kv_heads, heads // num_kv_heads).transpose(0, 1)
    return DistanceBias(by_distance.float().contiguous(), (by_distance * 1.4426950408889634).float().contiguous())
