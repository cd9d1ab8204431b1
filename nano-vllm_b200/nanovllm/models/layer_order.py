"""Execution order of the layers of a model that repeats a run of them."""
from __future__ import annotations


def layer_runs(num_layers: int, loop: dict | None) -> list[tuple[int, int, bool]]:
    """Execution order: (layer, pass, whether a pass opens right before it).  Layers [start, stop) run `times` times in a row."""
    if not loop:
        return [(i, 0, False) for i in range(num_layers)]
    a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    if not (0 <= a < b <= num_layers) or times < 1:
        raise ValueError("loop: need 0 <= start < stop <= number of layers and times >= 1")
    runs = [(i, 0, False) for i in range(a)]
    for k in range(times):
        runs += [(i, k, i == a) for i in range(a, b)]
    return runs + [(i, 0, False) for i in range(b, num_layers)]
