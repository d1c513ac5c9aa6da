"""Tiny Dizepel configurations for the tests: sizes that share nothing with each other, every branch of the design."""


def rotation(dims, base, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def left(heads, kv_heads, dim, scale, conv, softcap=None, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "conv": conv}
    if softcap:
        m["softcap"] = softcap
    if rot:
        m["rot"] = rot
    return m


def right(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def layer(a, b, ff):
    return {"type": "parallel", "mixer": {"left": a, "right": b}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def model(vocab, width, eps, scale, taps, loop, layers):
    cfg = {"architecture": "Dizepel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
           "canon": {"taps": taps}, "layers": layers}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


CONFIGS = {
    # grouped kv heads, a low cap, stretched rotation of half a head; a span in the middle of the layers that runs three times; a
    # layer without feed-forward inside it; sizes that nothing divides
    "X": model(211, 72, 1e-5, 3.0, 4, (1, 3, 3), [
        layer(left(4, 2, 24, 0.25, 3, 6.0, rotation(12, 500.0, (4.0, 40, 4.0, 0.5))), right(6, 10, 12, 3, 2, 5), 100),
        layer(left(3, 3, 20, 0.3, 4, 30.0, rotation(20, 1.0e4)), right(5, 7, 33, 1, 4, 1), None),
        layer(left(6, 1, 12, 0.4, 2, None, rotation(6, 77.0, (8.0, 64, 8.0, 1.0))), right(2, 24, 9, 2, 3, 3), 36)]),
    # one kv head; no rotation; taps of one and of more than four; a span of one layer at the end; no cap
    "Y": model(130, 64, 1e-6, 1.0, 2, (1, 2, 2), [
        layer(left(5, 1, 16, 0.4, 6), right(3, 8, 20, 3, 1, 4), 48),
        layer(left(2, 2, 40, 0.2, 1, 3.0), right(4, 16, 5, 2, 5, 2), 60)]),
    # head sizes of the tensor-core kernels, no span, a filter of one tap in front, states of several tiles
    "Z": model(300, 96, 1e-5, 9.5, 1, None, [
        layer(left(4, 1, 64, 0.2, 4, 12.0, rotation(32, 2.0e5, (16.0, 128, 16.0, 2.0))), right(4, 64, 16, 2, 4, 2), 72),
        layer(left(3, 3, 128, 0.09, 4, 40.0, rotation(128, 1.0e4)), right(2, 48, 128, 1, 4, 1), 56),
        layer(left(6, 2, 144, 0.08, 3, 20.0, rotation(16, 900.0)), right(8, 12, 24, 4, 3, 8), 40)]),
}
BLOCK = {"X": 8, "Y": 16, "Z": 16}
