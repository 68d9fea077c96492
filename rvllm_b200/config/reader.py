"""Reading numbers out of nested config.json objects: every problem is collected, none raises on its own."""
from __future__ import annotations

from typing import List


def is_int(v) -> bool:
    return isinstance(v, int) and not isinstance(v, bool)


def is_num(v) -> bool:
    return isinstance(v, (int, float)) and not isinstance(v, bool)


class NumberReader:
    """`problems` lists what was wrong; a number that could not be read is replaced by a harmless one."""

    def __init__(self):
        self.problems: List[str] = []

    def integer(self, d, key, what, minimum=1):
        v = d.get(key) if isinstance(d, dict) else None
        if not is_int(v) or v < minimum:
            self.problems.append(f"{what}`{key}` must be an integer >= {minimum}, got {v!r}")
            return max(minimum, 1)
        return v

    def number(self, d, key, what, positive=True):
        v = d.get(key) if isinstance(d, dict) else None
        if not is_num(v) or (positive and not v > 0):
            self.problems.append(f"{what}`{key}` must be a number{' > 0' if positive else ''}, got {v!r}")
            return 1.0
        return float(v)
