"""The run order of designs whose config.json names a run of layers that repeats:
`loop` = {`start`, `stop`, `times`}: the layers start .. stop - 1 run `times` times in a row with
the same weights, each pass a copy with keys and state of its own; row t of the model's table
`LOOP_VECTORS` is added to the residual before pass t.  `embedding_again`: the embedding's output
is added to it before every pass but the first, ahead of the row.  `project`: instead of the rows of
`LOOP_VECTORS`, every pass begins with x <- W [x; embedding's output], W the model's matrix
`LOOP_MATRIX`."""
from __future__ import annotations

from typing import Any, Mapping

from ..config.model_config import ConfigError, KeyReader, RunEntry

LOOP_VECTORS = "loop_step"      # the model's table of the vectors added before each pass
LOOP_MATRIX = "loop_in"         # the model's matrix that the rows go through before each pass


def _count(raw: Mapping[str, Any], key: str, where: str) -> int:
    v = raw.get(key)
    if isinstance(v, bool) or not isinstance(v, int) or v < 0:
        raise ConfigError(f"{where}: {key!r} must be a non-negative integer, got {v!r}")
    return v


def looped_run_order(raw: Mapping[str, Any], n_layers: int, embedding_again: bool = False, project: bool = False):
    """(run order, number of passes: 0 without a `loop`)."""
    loop = raw.get("loop")
    if loop is None:
        return tuple(RunEntry(layer=i) for i in range(n_layers)), 0
    where = "config.json loop"
    if not isinstance(loop, dict):
        raise ConfigError(f"{where}: must be an object")
    start, stop = _count(loop, "start", where), _count(loop, "stop", where)
    times = KeyReader(loop, where).integer("times")
    if not start <= stop <= n_layers:
        raise ConfigError(f"{where}: 'start' <= 'stop' <= the number of layers, got {start} and {stop}")
    if start == stop:
        # an empty run: nothing repeats and no vector is ever added (the table is still the model's)
        return tuple(RunEntry(layer=i) for i in range(n_layers)), times
    order = [RunEntry(layer=i) for i in range(start)]
    for t in range(times):
        order += [RunEntry(layer=i, copy=t, add=(LOOP_VECTORS, t) if i == start and not project else None,
                           project=LOOP_MATRIX if i == start and project else None,
                           add_embedding=embedding_again and i == start and t > 0)
                  for i in range(start, stop)]
    order += [RunEntry(layer=i) for i in range(stop, n_layers)]
    return tuple(order), times
