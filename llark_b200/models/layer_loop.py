"""A `loop` over part of a layer list, as native decoders' configurations carry it: {start, stop, times}, the layers start ..
stop - 1 run `times` times in a row on the same weights, every pass with a cache or state of its own."""


def read_loop(entry, n_layers):
    """The validated loop of a configuration; None when there is none (or when it names no layer)."""
    if not entry:
        return None
    loop = {k: int(entry[k]) for k in ("start", "stop", "times")}
    if not (0 <= loop["start"] <= loop["stop"] <= n_layers) or loop["times"] < 1:
        raise ValueError("loop must name a range of layers and a positive number of passes")
    return None if loop["start"] == loop["stop"] else loop


def layer_runs(loop, n_layers):
    """(layer, pass, first layer of a pass?) in the order the layers run; pass is None outside the loop."""
    if loop is None:
        return [(i, None, False) for i in range(n_layers)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, None, False) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t, i == a) for i in range(a, b)]
    return runs + [(i, None, False) for i in range(b, n_layers)]
