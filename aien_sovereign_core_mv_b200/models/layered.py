"""What the readers of configurations that list their layers one by one share: checked access to keys, a stretch of layers
that runs several times, the stop tokens."""
from __future__ import annotations

from typing import Any, Mapping, Optional, Tuple

from ..config.model_config import ConfigError


def need(obj: Any, key: str, where: str, kind=None):
    if not isinstance(obj, Mapping) or key not in obj or obj[key] is None:
        raise ConfigError(f"config.json: {where}.{key} is missing")
    v = obj[key]
    if kind is int:
        if isinstance(v, bool) or not isinstance(v, int) or v <= 0:
            raise ConfigError(f"config.json: {where}.{key} must be a positive integer, got {v!r}")
    elif kind is float:
        if isinstance(v, bool) or not isinstance(v, (int, float)):
            raise ConfigError(f"config.json: {where}.{key} must be a number, got {v!r}")
        v = float(v)
    return v


def opt_number(obj: Any, key: str, default: float, where: str = "config") -> float:
    v = obj.get(key) if isinstance(obj, Mapping) else None
    if v is None:
        return float(default)
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"config.json: {where}.{key} must be a number, got {v!r}")
    return float(v)


def opt_count(obj: Any, key: str, default: int, where: str) -> int:
    v = obj.get(key) if isinstance(obj, Mapping) else None
    if v is None:
        return int(default)
    if isinstance(v, bool) or not isinstance(v, int) or v < 0:
        raise ConfigError(f"config.json: {where}.{key} must be a non-negative integer, got {v!r}")
    return int(v)


def run_order(num_layers: int, loop: Optional[Tuple[int, int, int]]):
    """[(layer, pass number that this run opens or -1)]: layers start .. stop - 1 run ``times`` times in a row."""
    if loop is None:
        return [(i, -1) for i in range(num_layers)]
    start, stop, times = loop
    order = [(i, -1) for i in range(start)]
    for t in range(times):
        order += [(i, t if i == start else -1) for i in range(start, stop)]
    return order + [(i, -1) for i in range(stop, num_layers)]


def read_loop(raw: Mapping[str, Any], num_layers: int) -> Optional[Tuple[int, int, int]]:
    loop = raw.get("loop")
    if loop is None:
        return None
    start, stop = opt_count(loop, "start", 0, "loop"), need(loop, "stop", "loop", int)
    times = need(loop, "times", "loop", int) if loop.get("times") is not None else 1
    if not (0 <= start < stop <= num_layers):
        raise ConfigError(f"config.json: loop.start {start} and loop.stop {stop} must name a stretch of the {num_layers} layers")
    return start, stop, times


def read_layers(raw: Mapping[str, Any]):
    layers = need(raw, "layers", "config")
    if not isinstance(layers, (list, tuple)) or not layers:
        raise ConfigError("config.json: layers must be a non-empty list")
    return layers


def read_eos(generation_config: Optional[Mapping[str, Any]], raw: Mapping[str, Any]) -> Tuple[int, ...]:
    for source in (generation_config, raw):
        v = source.get("eos_token_id") if isinstance(source, Mapping) else None
        if v is not None:
            return tuple(int(t) for t in (v if isinstance(v, (list, tuple)) else [v]))
    return ()
