"""A plain, slow implementation of the Dizepel design on whole sequences: one function per mechanism, float64 or float32
on the CPU, no cache, no batching, nothing shared with the package.  The tests compare the engine with it.

A model is (config dict, {tensor name: tensor}).  Notation: T tokens, D width, x the residual stream [T, D].
"""
import math

import torch


def by_rms(x, eps):
    """x divided by the root of its mean square over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    """x less its mean, divided by its standard deviation, times a weight; no bias."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z / (1 + torch.exp(-z))


def causal_filter(u, w):
    """u [T, C], w [C, taps]: sum over j of w[:, j] * u at (t - taps + 1 + j), nothing before the first token."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * u[:T - back]
    return y


def poly_norm(z, coef, eps):
    """a N(z) + b N(z^2) + c N(z^3) + e, each power divided by its own root mean square over the row."""
    a, b, c, e = coef
    return a * by_rms(z, eps) + b * by_rms(z ** 2, eps) + c * by_rms(z ** 3, eps) + e


def rotary_frequencies(rot):
    """(frequencies, what cos and sin are multiplied by) of a rotation of rot["dims"] values, stretched if asked."""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    pair_at = lambda turns: n * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(pair_at(sc["fast"])), 0), min(math.ceil(pair_at(sc["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * r + fi * (1 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1


def rotate_halves(x, positions, rot):
    """x [T, heads, d]: of the first rot["dims"] = n values, i and i + n/2 turn by position * frequency_i; the rest passes."""
    if not rot:
        return x
    f, mult = rotary_frequencies(rot)
    n = rot["dims"]
    ang = positions.to(x.dtype)[:, None, None] * torch.tensor(f, dtype=x.dtype)
    c, s = torch.cos(ang) * mult, torch.sin(ang) * mult
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., n:]], -1)


def cap_scores(s, cap):
    return cap * torch.tanh(s / cap) if cap else s


def softmax_with_sink(s, seen, sink):
    """Rows of s over the keys that `seen` allows; exp(sink) joins the denominator without a key or a value."""
    s = s.masked_fill(~seen, float("-inf"))
    m = torch.maximum(s.max(-1, keepdim=True).values, sink)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - m))


# ---------------------------------------------------------------------------------------------------- mixers

def attention(h, W, m):
    """Grouped heads whose queries and keys pass a short filter over time; the values are the filtered keys before they are
    rotated; capped scores; a learned sink per head."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = causal_filter(h @ W["q"].T + W["q.b"], W["q.conv"]).reshape(T, H, d)
    k = causal_filter(h @ W["k"].T + W["k.b"], W["k.conv"]).reshape(T, G, d)
    v = k
    pos = torch.arange(T)
    q, k = rotate_halves(q, pos, m.get("rot")), rotate_halves(k, pos, m.get("rot"))
    seen = pos[None, :] <= pos[:, None]
    out = torch.zeros(T, H, d, dtype=h.dtype)
    for hd in range(H):
        g = hd // (H // G)
        s = cap_scores((q[:, hd] @ k[:, g].T) * m["scale"], m.get("softcap"))
        out[:, hd] = softmax_with_sink(s, seen, W["sink"][hd]) @ v[:, g]
    return out.reshape(T, H * d) @ W["o"].T


def state_space(h, W, m, eps):
    """A matrix per head that decays by a scalar per token, takes in B x^T and is read with C; the gate comes before the norm."""
    T, H, dv, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    p = h @ W["in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_filter(xbc, W["conv"]) + W["conv.b"])
    x = xbc[:, :inner].reshape(T, H, dv)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N).repeat_interleave(H // G, 1)
    C = xbc[:, inner + G * N:].reshape(T, G, N).repeat_interleave(H // G, 1)
    a = dt + W["dt_bias"]
    step = torch.where(a > 0, a, torch.zeros_like(a)) + torch.log1p(torch.exp(-a.abs()))
    decay = torch.exp(-torch.exp(W["A_log"]) * step)
    S = torch.zeros(H, N, dv, dtype=h.dtype)
    y = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        S = decay[t][:, None, None] * S + step[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        y[t] = (S * C[t][:, :, None]).sum(1) + W["D"][:, None] * x[t]
    y = y.reshape(T, inner) * silu(z)
    parts = m.get("norm_groups", 1)
    y = by_rms(y.reshape(T, parts, inner // parts), eps).reshape(T, inner) * W["norm"]
    return y @ W["o"].T


def parallel_mixer(h, W, m, eps):
    left = attention(h, sub(W, "left."), m["left"])
    right = state_space(h, sub(W, "right."), m["right"], eps)
    return 0.5 * (by_rms(left, eps) * W["left.out"] + by_rms(right, eps) * W["right.out"])


def feed_forward(h, W, eps):
    return poly_norm(h @ W["up"].T, W["act"], eps) @ W["down"].T


# ---------------------------------------------------------------------------------------------------- the model

def sub(W, prefix):
    return {n[len(prefix):]: t for n, t in W.items() if n.startswith(prefix)}


def layer(x, W, L, eps):
    h = centred_norm(x, W["norm1"], eps)
    h = h + causal_filter(h, W["canon1"])
    x = x + centred_norm(parallel_mixer(h, sub(W, "mix."), L["mixer"], eps), W["norm1b"], eps)
    if L.get("mlp"):
        h = centred_norm(x, W["norm2"], eps)
        h = h + causal_filter(h, W["canon2"])
        x = x + centred_norm(feed_forward(h, sub(W, "mlp."), eps), W["norm2b"], eps)
    return x


def layer_runs(cfg):
    """(layer, pass that starts here or None) in the order in which they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop") or {"start": 0, "stop": 0, "times": 0}
    a, b = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(a)]
    for t in range(loop["times"] if b > a else 0):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def forward(cfg, weights, tokens, dtype=torch.float64, streams=None):
    """Logits [T, vocab]; `streams`: a list that receives the stream after every layer run."""
    W = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i, start in layer_runs(cfg):
        if start is not None:
            x = x + W["loop.step"][start]
        x = layer(x, sub(W, f"l{i}."), cfg["layers"][i], eps)
        if streams is not None:
            streams.append(x.clone())
    return centred_norm(x, W["final.norm"], eps) @ W["head"].T


def tensor_shapes(cfg):
    """{name: shape} of every tensor of a model."""
    D, V, taps = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]
    out = {"embed": (V, D), "final.norm": (D,), "head": (V, D)}
    loop = cfg.get("loop")
    if loop and loop["stop"] > loop["start"]:
        out["loop.step"] = (loop["times"], D)
    for i, L in enumerate(cfg["layers"]):
        p, a, b = f"l{i}.", L["mixer"]["left"], L["mixer"]["right"]
        H, G, d, inner = a["heads"], a["kv_heads"], a["dim"], b["heads"] * b["vdim"]
        ch = inner + 2 * b["groups"] * b["state"]
        out.update({p + n: (D,) for n in ("norm1", "norm1b")})
        out[p + "canon1"] = (D, taps)
        l, r = p + "mix.left.", p + "mix.right."
        out.update({l + "q": (H * d, D), l + "q.b": (H * d,), l + "k": (G * d, D), l + "k.b": (G * d,), l + "q.conv": (H * d, a["conv"]),
                    l + "k.conv": (G * d, a["conv"]), l + "sink": (H,), l + "o": (D, H * d), l + "out": (D,)})
        out.update({r + "in": (inner + ch + b["heads"], D), r + "conv": (ch, b["conv"]), r + "conv.b": (ch,), r + "dt_bias": (b["heads"],),
                    r + "A_log": (b["heads"],), r + "D": (b["heads"],), r + "norm": (inner,), r + "o": (D, inner), r + "out": (D,)})
        if L.get("mlp"):
            f = L["mlp"]["ff"]
            out.update({p + "norm2": (D,), p + "norm2b": (D,), p + "canon2": (D, taps), p + "mlp.up": (f, D), p + "mlp.down": (D, f),
                        p + "mlp.act": (4,)})
    return out


def random_weights(cfg, seed, std=None, dtype=torch.float32):
    """Weights whose every part matters: matrices of about unit gain, norm weights around one, filters and biases of the size of
    what they join, decays from slow to fast."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        t = torch.randn(*shape, generator=g)
        last = name.split(".")[-1]
        if last in ("norm", "norm1", "norm2", "norm1b", "norm2b", "out"):
            t = 1 + 0.3 * t
        elif last in ("canon1", "canon2", "conv"):
            t = t * 0.5
        elif last == "A_log":
            t = torch.log(0.05 + 2 * torch.rand(*shape, generator=g))
        elif last == "dt_bias":
            t = t - 1
        elif last in ("D", "sink", "act"):
            pass
        elif last == "step" or name == "embed":
            pass
        elif len(shape) == 1:
            t = t * 0.5                                              # biases
        else:
            t = t * (std if std is not None else 1.0 / math.sqrt(shape[1]))
        out[name] = t.to(dtype)
    return out
