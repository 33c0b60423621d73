"""Checked reading of ``config.json`` entries: an integer, a positive number, an object, or one error that names the place."""
from __future__ import annotations

import math

from ..errors import BadFormat


def integer(d: dict, key: str, where: str, minimum: int = 1) -> int:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, int):
        raise BadFormat(f'config.json: {where} needs an integer "{key}", not {v!r}')
    if v < minimum:
        raise BadFormat(f'config.json: {where}: "{key}" is {v}, expected at least {minimum}')
    return v


def number(d: dict, key: str, where: str, default: float = None) -> float:
    """A positive number; ``default`` (if given) where the entry is absent or null."""
    v = d.get(key)
    if v is None and default is not None:
        return default
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not math.isfinite(v) or v <= 0:
        raise BadFormat(f'config.json: {where} needs a positive number "{key}", not {v!r}')
    return float(v)


def obj(d: dict, key: str, where: str) -> dict:
    v = d.get(key)
    if not isinstance(v, dict):
        raise BadFormat(f'config.json: {where} needs an object "{key}", not {v!r}')
    return v
