"""A plain, slow implementation of the Fivedra design on whole sequences: one function per mechanism, float64 or
float32 on the CPU, no cache, no batching, nothing shared with the package.  The tests compare the engine with it.

A model is (config dict, {tensor name: tensor}).  Notation: T tokens, D width, x the residual stream [T, D].
"""
import math

import torch


def rms(x, eps):
    """x divided by the root of its mean square over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x, w, eps):
    """The norm whose stored weight is the distance from one."""
    return rms(x, eps) * (1 + w)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def log_sigmoid(z):
    return torch.where(z >= 0, -torch.log1p(torch.exp(-z.abs())), z - torch.log1p(torch.exp(-z.abs())))


def bucket(n, count, far):
    """Which of `count` entries of a distance table a distance n >= 0 reads: the first half one by one, the rest by the
    logarithm of the distance, so that `far` and everything beyond it is the last."""
    half = count // 2
    if n < half:
        return n
    return min(count - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (count - half)))


def rotary_frequencies(rot):
    """(frequencies, what cos and sin are multiplied by) of a rotation of rot["dims"] values, stretched if asked."""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    at = lambda turns: n * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(at(sc["fast"])), 0), min(math.ceil(at(sc["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * r + fi * (1 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1


def rotate_neighbours(x, positions, rot):
    """x [T, ..., n]: the values 2i and 2i + 1 of the first rot["dims"] turn by position * frequency_i; the rest passes."""
    f, mult = rotary_frequencies(rot)
    n = rot["dims"]
    ang = positions.to(x.dtype).reshape(-1, *([1] * (x.dim() - 1))) * torch.tensor(f, dtype=x.dtype)
    c, s = torch.cos(ang) * mult, torch.sin(ang) * mult
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    y = torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)
    return torch.cat([y, x[..., n:]], -1)


def softmax_with_sink(s, seen, sink):
    """Rows of s over the keys that `seen` allows; exp(sink) joins the denominator without a key or a value."""
    s = s.masked_fill(~seen, float("-inf"))
    m = torch.maximum(s.max(-1, keepdim=True).values, torch.as_tensor(float(sink), dtype=s.dtype))
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - m))


# ---------------------------------------------------------------------------------------------------- mixers

def min_gru_mixer(h, W):
    """A gated recurrence element by element; gate and candidate read the current token only."""
    z = sigmoid(h @ W["z"].T + W["z.b"])
    u = h @ W["x"].T + W["x.b"]
    cand = torch.where(u >= 0, u + 0.5, sigmoid(u))
    g = h @ W["g"].T
    S = torch.zeros(z.shape[1], dtype=h.dtype)
    rows = []
    for t in range(h.shape[0]):
        S = (1 - z[t]) * S + z[t] * cand[t]
        rows.append(S * (g[t] * sigmoid(g[t])))
    return torch.stack(rows) @ W["o"].T


def window_attention(h, W, m):
    """Grouped heads whose keys are their values, a learned bias per distance bucket and head, a sliding window and
    one more in the softmax's denominator."""
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ W["q"].T + W["q.b"]).reshape(T, H, d)
    k = (h @ W["k"].T + W["k.b"]).reshape(T, G, d)
    table = W["rel"]
    which = torch.tensor([bucket(n, table.shape[0], m["bias_max"]) for n in range(T)])
    pos = torch.arange(T)
    dist = pos[:, None] - pos[None, :]
    seen = dist >= 0
    size = (m.get("mask") or {}).get("size")
    if size:
        seen = seen & (dist < size)
    out = torch.zeros(T, H, d, dtype=h.dtype)
    for hd in range(H):
        kk = k[:, hd // (H // G)]
        s = (q[:, hd] @ kk.T) * m["scale"] + table[which[dist.clamp(min=0)], hd]
        out[:, hd] = softmax_with_sink(s, seen, torch.zeros((), dtype=h.dtype)) @ kk
    return out.reshape(T, H * d) @ W["o"].T


def matrix_memory(h, W, m, eps):
    """A matrix per head that every token decays, writes k v^T into and reads with q; exponential gates kept in range by a
    running maximum; a norm per head and a sigmoid gate per value."""
    T = h.shape[0]
    H, dk, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ W["q"].T).reshape(T, H, dk) * dk ** -0.5
    k = (h @ W["k"].T).reshape(T, H, dk)
    v = (h @ W["v"].T).reshape(T, H, dv)
    li = cap * torch.tanh((h @ W["i"].T + W["i.b"]) / cap)
    lf = log_sigmoid(cap * torch.tanh((h @ W["f"].T + W["f.b"]) / cap))
    S, n = torch.zeros(H, dk, dv, dtype=h.dtype), torch.zeros(H, dk, dtype=h.dtype)
    top = torch.zeros(H, dtype=h.dtype)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        new = torch.maximum(lf[t] + top, li[t])
        keep, write = torch.exp(lf[t] + top - new), torch.exp(li[t] - new)
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        top = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-top)) + 1e-6
        out[t] = (S * q[t][:, :, None]).sum(1) / den[:, None]
    y = rms(out, eps).reshape(T, H * dv) * W["norm"] * sigmoid(h @ W["g"].T)
    return y @ W["o"].T


def parallel_mixer(h, W, m, eps):
    left = window_attention(h, sub(W, "left."), m["left"])
    right = matrix_memory(h, sub(W, "right."), m["right"], eps)
    return m["left_scale"] * left + m["right_scale"] * right


def latent_attention_mixer(h, W, m, eps):
    """Queries, keys and values expanded from normed low-rank vectors; one rotated key part that all heads share; every
    earlier token is seen; a learned sink per head."""
    T = h.shape[0]
    H, dk, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    cq = rms(h @ W["dq"].T, eps) * W["dq.norm"]
    q = (cq @ W["uq"].T).reshape(T, H, dk + dr)
    q_plain, q_rot = q[..., :dk], rotate_neighbours(q[..., dk:], pos, m["rot"])
    d = h @ W["dkv"].T
    c = rms(d[:, :r], eps) * W["dkv.norm"]
    k_rot = rotate_neighbours(d[:, r:], pos, m["rot"])
    k_plain = (c @ W["uk"].T).reshape(T, H, dk)
    v = (c @ W["uv"].T).reshape(T, H, dv)
    seen = pos[None, :] <= pos[:, None]
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for hd in range(H):
        s = (q_plain[:, hd] @ k_plain[:, hd].T + q_rot[:, hd] @ k_rot.T) * m["scale"]
        out[:, hd] = softmax_with_sink(s, seen, W["sink"][hd]) @ v[:, hd]
    return out.reshape(T, H * dv) @ W["o"].T


def squared_relu_feed_forward(h, W):
    return torch.relu(h @ W["up"].T) ** 2 @ W["down"].T


# ---------------------------------------------------------------------------------------------------- the model

def sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def mixer(kind, h, W, m, eps):
    if kind == "mingru":
        return min_gru_mixer(h, W)
    if kind == "parallel":
        return parallel_mixer(h, W, m, eps)
    return latent_attention_mixer(h, W, m, eps)


def layer(x, cfg, weights, i):
    """Both branches read the same x, each through a norm of its own, and are added together."""
    L, eps, p = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}."
    y = mixer(L["type"], zero_centred_norm(x, weights[p + "norm1"], eps), sub(weights, p + "mix."), L["mixer"], eps)
    if L.get("mlp"):
        y = y + squared_relu_feed_forward(zero_centred_norm(x, weights[p + "norm2"], eps), sub(weights, p + "mlp."))
    return x + y


def forward(cfg, weights, tokens, dtype=torch.float64, streams=None):
    """Logits [T, vocab] of one whole sequence.  `streams`: a list that receives x after every layer."""
    W = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    for i in range(len(cfg["layers"])):
        x = layer(x, cfg, W, i)
        if streams is not None:
            streams.append(x)
    return zero_centred_norm(x, W["final.norm"], cfg["norm"]["eps"]) @ W["head"].T


def tensor_shapes(cfg):
    """{tensor name: shape} of a model of this configuration; a parallel layer's `rel` has `left["buckets"]` rows (a key
    of the tests' own configurations: the engine reads the number from the tensor)."""
    D, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, D), "final.norm": (D,), "head": (V, D)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        x = p + "mix."
        s[p + "norm1"] = (D,)
        if L["type"] == "mingru":
            w = m["width"]
            s.update({x + "z": (w, D), x + "z.b": (w,), x + "x": (w, D), x + "x.b": (w,), x + "g": (w, D), x + "o": (D, w)})
        elif L["type"] == "latent_attention":
            H, dk, dr, dv, r, rq = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            s.update({x + "dq": (rq, D), x + "dq.norm": (rq,), x + "uq": (H * (dk + dr), rq), x + "dkv": (r + dr, D),
                      x + "dkv.norm": (r,), x + "uk": (H * dk, r), x + "uv": (H * dv, r), x + "sink": (H,),
                      x + "o": (D, H * dv)})
        else:
            a, b = m["left"], m["right"]
            H, G, d = a["heads"], a["kv_heads"], a["dim"]
            s.update({x + "left.q": (H * d, D), x + "left.q.b": (H * d,), x + "left.k": (G * d, D), x + "left.k.b": (G * d,),
                      x + "left.rel": (a.get("buckets", 16), H), x + "left.o": (D, H * d)})
            H, dk, dv = b["heads"], b["dim"], b["vdim"]
            s.update({x + "right.q": (H * dk, D), x + "right.k": (H * dk, D), x + "right.v": (H * dv, D),
                      x + "right.g": (H * dv, D), x + "right.o": (D, H * dv), x + "right.norm": (H * dv,),
                      x + "right.i": (H, D), x + "right.i.b": (H,), x + "right.f": (H, D), x + "right.f.b": (H,)})
        f = L.get("mlp")
        if f:
            s[p + "norm2"] = (D,)
            s.update({p + "mlp.up": (f["ff"], D), p + "mlp.down": (D, f["ff"])})
    return s


def random_weights(cfg, seed=0, std=None, dtype=torch.bfloat16):
    """Weights whose branches all matter: matrices of standard deviation 1 / sqrt(columns) (or `std`), norm weights around
    their neutral value, gates around one half, forget gates that keep most of the state, sinks and biases of a size that
    changes the softmax."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in tensor_shapes(cfg).items():
        r = torch.randn(shape, generator=g)
        if name.endswith("norm1") or name.endswith("norm2") or name == "final.norm":
            t = 0.2 * r
        elif name.endswith(".norm"):
            t = 1 + 0.2 * r
        elif name.endswith(".f.b"):
            t = 2.0 + 1.5 * r
        elif name.endswith(".z.b"):
            t = -1.0 + r
        elif name.endswith(".i.b") or name.endswith(".b"):
            t = 0.3 * r
        elif name.endswith(".sink") or name.endswith(".rel"):
            t = r
        elif name == "embed":
            t = r / cfg["embedding"]["scale"]
        else:
            t = r * (std if std is not None else 1.0 / math.sqrt(shape[-1]))
        W[name] = t.to(dtype)
    return W
