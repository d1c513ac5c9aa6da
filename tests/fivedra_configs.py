"""Tiny Fivedra configurations for the tests: sizes that share nothing with each other, every branch of the design."""


def mingru(width):
    return {"type": "mingru", "mixer": {"width": width}}


def window(heads, kv_heads, dim, scale, bias_max, size=None, buckets=16):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "bias_max": bias_max, "buckets": buckets}
    if size:
        m["mask"] = {"size": size}
    return m


def memory(heads, dim, vdim, cap=15.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def parallel(left, right, left_scale=1.0, right_scale=1.0):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}}


def rotation(dims, base, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, rot):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                                  "q_rank": q_rank, "scale": scale, "rot": rot}}


def with_mlp(layer, ff):
    return dict(layer, mlp={"kind": "dense", "ff": ff} if ff else None)


def model(vocab, width, eps, scale, layers):
    return {"architecture": "Fivedra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": layers}


CONFIGS = {
    # grouped kv heads; a window shorter than where the buckets end and one longer; a layer without feed-forward; factors of
    # both signs; head and value sizes that nothing divides; an odd number of buckets
    "X": model(211, 72, 1e-5, 3.0, [
        with_mlp(parallel(window(4, 2, 24, 0.25, 60, 21), memory(3, 10, 18, 4.0), 0.7, -1.3), 100),
        with_mlp(mingru(50), 60),
        with_mlp(latent(3, 20, 12, 14, 40, 28, 0.2, rotation(12, 500.0, (4.0, 40, 4.0, 0.5))), None),
        with_mlp(parallel(window(2, 2, 12, 0.3, 13, 50, 7), memory(1, 33, 70, 9.0), -0.4, 2.0), 36)]),
    # one kv head; no window; the recurrent layer last and first; a rotation that is not stretched
    "Y": model(130, 64, 1e-6, 1.0, [
        with_mlp(mingru(37), None),
        with_mlp(parallel(window(6, 1, 16, 0.4, 200, None, 32), memory(2, 8, 4, 1.5), 1.0, 1.0), 48),
        with_mlp(latent(2, 16, 4, 40, 16, 8, 0.3, rotation(4, 10000.0)), 20),
        with_mlp(mingru(96), 64)]),
    # head sizes of the tensor-core kernels, windows longer than a tile, values wider than a block of the memory's columns
    "Z": model(300, 96, 1e-5, 9.5, [
        with_mlp(latent(4, 32, 16, 24, 80, 40, 0.15, rotation(16, 2.0e5, (16.0, 128, 16.0, 2.0))), 40),
        with_mlp(parallel(window(4, 1, 64, 0.125, 96, 150), memory(2, 64, 130), 0.5, 0.8), 72),
        with_mlp(parallel(window(3, 3, 128, 0.09, 400, 129, 24), memory(4, 24, 64, 2.0), 1.5, 0.3), 56),
        with_mlp(mingru(128), 88)]),
}
BLOCK = {"X": 8, "Y": 16, "Z": 16}
