"""Reading typed values out of a config.json with errors that name the key; shared by the configuration readers."""
from __future__ import annotations

from typing import Mapping

from .errors import ConfigError


def need(raw, key: str, where: str):
    if not isinstance(raw, Mapping) or key not in raw or raw[key] is None:
        raise ConfigError(f"config.json lacks '{where}{key}'")
    return raw[key]


def integer(raw, key: str, where: str, least: int = 1) -> int:
    v = need(raw, key, where)
    if isinstance(v, bool) or not isinstance(v, int) or v < least:
        raise ConfigError(f"config key '{where}{key}' must be an integer >= {least}, got {v!r}")
    return v


def number(raw, key: str, where: str, positive: bool = False) -> float:
    v = need(raw, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or (positive and not v > 0):
        raise ConfigError(f"config key '{where}{key}' must be a{' positive' if positive else ''} number, got {v!r}")
    return float(v)
