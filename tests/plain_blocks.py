"""Plain, slow implementation of the block models (config.json + model.safetensors directories) in numpy.

Test oracle only: one function per mechanism, token by token where the mechanism is a recurrence, whole sequence at once
otherwise.  It shares no code with the library (not even the file readers) and computes in binary64 unless told otherwise.
"""
import json
import struct

import numpy as np


# ------------------------------------------------------------------ files
def read_safetensors(path, dtype=np.float64):
    with open(path, "rb") as f:
        raw = f.read()
    n = struct.unpack("<Q", raw[:8])[0]
    head = json.loads(raw[8:8 + n])
    out = {}
    for name, t in head.items():
        if name == "__metadata__":
            continue
        lo, hi = t["data_offsets"]
        b = raw[8 + n + lo:8 + n + hi]
        if t["dtype"] == "BF16":
            a = (np.frombuffer(b, np.uint16).astype(np.uint32) << 16).view(np.float32).astype(dtype)
        elif t["dtype"] == "F32":
            a = np.frombuffer(b, np.float32).astype(dtype)
        else:
            raise ValueError(t["dtype"])
        out[name] = a.reshape(t["shape"])
    return out


def to_bf16_bits(a):
    """float array -> bfloat16 bit patterns, round to nearest even (finite values)."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32).astype(np.uint64)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def write_safetensors(path, tensors):
    """{name: float array} -> bfloat16 safetensors file."""
    head, blobs, off = {}, [], 0
    for name, a in tensors.items():
        b = to_bf16_bits(a).tobytes()
        head[name] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [off, off + len(b)]}
        blobs.append(b)
        off += len(b)
    h = json.dumps(head).encode()
    h += b" " * (-len(h) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))


# ------------------------------------------------------------------ elementary functions
def sigmoid(z):
    return np.where(z >= 0, 1 / (1 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def unit_rms(x, eps):
    """Last axis divided by its root mean square."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_around_zero(x, w, eps):
    return unit_rms(x, eps) * (1 + w)


def norm(x, w, eps):
    return unit_rms(x, eps) * w


# ------------------------------------------------------------------ embedding
def embed(tokens, W, cfg):
    e = cfg["embedding"]
    x = W["embed"][tokens] * e.get("scale", 1.0)
    b = e.get("bigram")
    if b:
        rows = [b["buckets"]] + [(int(p) * b["mul_prev"] + int(t) * b["mul_cur"]) % b["buckets"] for p, t in zip(tokens[:-1], tokens[1:])]
        x = x + W["bigram"][rows]
    return x


# ------------------------------------------------------------------ mixers (h: [tokens, width])
def rotate_half(x, positions, base, dims):
    """x [tokens, heads, dim]: dimensions 0 .. dims-1 in the pairing (i, i + dims/2)."""
    out = x.copy()
    half = dims // 2
    f = base ** (-2.0 * np.arange(half) / dims)
    a = positions[:, None] * f[None, :]
    c, s = np.cos(a)[:, None, :].astype(x.dtype), np.sin(a)[:, None, :].astype(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def window_pool_attention(h, W, p, m):
    """Causal sliding window plus one mean key / value per block that lies wholly before the window."""
    T = h.shape[0]
    H, G, D, DV = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T).reshape(T, H, D)
    k = (h @ W[p + "k"].T).reshape(T, G, D)
    v = (h @ W[p + "v"].T).reshape(T, G, DV)
    size, pool = m["mask"]["size"], m["mask"]["pool"]
    nb = T // pool
    kp = k[:nb * pool].reshape(nb, pool, G, D).mean(1)
    vp = v[:nb * pool].reshape(nb, pool, G, DV).mean(1)
    out = np.zeros((T, H, DV), h.dtype)
    for i in range(T):
        lo = max(0, i - size + 1)
        n_seen = max(0, min(nb, (i - size + 1) // pool)) if i - size + 1 > 0 else 0  # blocks b with b*pool + pool - 1 <= i - size
        for hd in range(H):
            g = hd // (H // G)
            keys = np.concatenate([kp[:n_seen, g], k[lo:i + 1, g]])
            vals = np.concatenate([vp[:n_seen, g], v[lo:i + 1, g]])
            s = keys @ q[i, hd] * m["scale"]
            e = np.exp(s - s.max())
            out[i, hd] = (e / e.sum()) @ vals
    return out.reshape(T, H * DV) @ W[p + "o"].T


def retention(h, W, p, m, eps):
    T = h.shape[0]
    H, D, DV = m["heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T).reshape(T, H, D)
    k = (h @ W[p + "k"].T).reshape(T, H, D)
    v = (h @ W[p + "v"].T).reshape(T, H, DV)
    pos = np.arange(T).astype(np.float64)
    if m.get("rot"):
        q, k = (rotate_half(a, pos, m["rot"]["base"], m["rot"]["dims"]) for a in (q, k))
    k = k * D ** -0.5
    S = np.zeros((H, D, DV), h.dtype)
    dec = np.array(m["decay"], h.dtype)[:, None, None]
    o = np.zeros((T, H, DV), h.dtype)
    for t in range(T):
        S = dec * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    o = unit_rms(o, eps).reshape(T, H * DV) * silu(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def parallel(h, W, p, m, eps):
    return m["left_scale"] * window_pool_attention(h, W, p + "left.", m["left"]) + m["right_scale"] * retention(h, W, p + "right.", m["right"], eps)


def wkv(h, W, p, m, eps):
    T = h.shape[0]
    H, D = m["heads"], m["dim"]
    hp = np.concatenate([np.zeros_like(h[:1]), h[:-1]])
    mix = {s: h + (hp - h) * W[p + "mu." + s] for s in "rkvgw"}
    r, k, v = ((mix[s] @ W[p + s].T).reshape(T, H, D) for s in "rkv")
    gate = silu(mix["g"] @ W[p + "g"].T)
    w = np.exp(-np.exp(np.tanh(mix["w"] @ W[p + "w1"].T) @ W[p + "w2"].T + W[p + "w0"])).reshape(T, H, D)
    u = W[p + "u"].reshape(H, D)
    S = np.zeros((H, D, D), h.dtype)
    o = np.zeros((T, H, D), h.dtype)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S + u[:, :, None] * kv, r[t])
        S = w[t][:, :, None] * S + kv
    o = unit_rms(o, eps).reshape(T, H * D) * W[p + "norm"] * gate
    return o @ W[p + "o"].T


def rotate_pairs(x, positions, base, dims):
    """x [tokens, heads, dim]: dimensions 0 .. dims-1 in the pairing (2i, 2i + 1)."""
    out = x.copy()
    for i in range(dims // 2):
        a = positions * base ** (-2.0 * i / dims)
        c, s = np.cos(a)[:, None].astype(x.dtype), np.sin(a)[:, None].astype(x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def window_softmax(q, k, v, scale, size, sink=None):
    """q, k [tokens, heads, dim], v [tokens, heads, vdim]: position i sees i - size + 1 .. i; sink [heads]: one more term
    exp(sink) of every denominator."""
    T, H, _ = q.shape
    out = np.zeros((T, H, v.shape[2]), q.dtype)
    for i in range(T):
        lo = max(0, i - size + 1)
        for hd in range(H):
            s = k[lo:i + 1, hd] @ q[i, hd] * scale
            top = s.max() if sink is None else max(s.max(), sink[hd])
            e = np.exp(s - top)
            out[i, hd] = e @ v[lo:i + 1, hd] / (e.sum() + (0 if sink is None else np.exp(sink[hd] - top)))
    return out


def latent_attention(h, W, p, m, eps):
    """Keys and values of every head from one normalised latent per token, and one rotated key part for all heads."""
    T = h.shape[0]
    H, D, R, DV, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T).astype(np.float64)
    q = (h @ W[p + "q"].T).reshape(T, H, D + R)
    down = h @ W[p + "dkv"].T
    c = norm(down[:, :C], W[p + "dkv.norm"], eps)
    turn = lambda a: rotate_pairs(a, pos, m["rot"]["base"], m["rot"]["dims"])  # noqa: E731
    q_rot, k_rot = turn(q[..., D:]), turn(down[:, None, C:])
    k = np.concatenate([(c @ W[p + "uk"].T).reshape(T, H, D), np.repeat(k_rot, H, axis=1)], axis=2)
    v = (c @ W[p + "uv"].T).reshape(T, H, DV)
    o = window_softmax(np.concatenate([q[..., :D], q_rot], axis=2), k, v, m["scale"], m["mask"]["size"], W[p + "sink"])
    o = o * sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(T, H * DV) @ W[p + "o"].T


MIXERS = {"parallel": parallel, "wkv": wkv, "latent_attention": latent_attention}


def feed_forward(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(h, W, p, top):
    """(experts, weights) of every token: the `top` largest scores sigmoid(z), which are the weights as they are."""
    z = h @ W[p + "router"].T
    pick = np.argsort(-z, axis=1, kind="stable")[:, :top]
    return pick, sigmoid(np.take_along_axis(z, pick, axis=1))


def experts(h, W, p, m):
    """A weight multiplies its expert's input."""
    pick, weight = route(h, W, p, m["router"]["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(pick[t], weight[t]):
            out[t] += feed_forward(w * h[t:t + 1], W, f"{p}e{e}.")[0]
    return out


# ------------------------------------------------------------------ the stack
def layer_runs(cfg):
    """Indices of the layers in the order they run (a looped range counts every pass)."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b, t = loop["start"], loop["stop"], loop["times"]
    return list(range(a)) + list(range(a, b)) * t + list(range(b, n))


def hyper_sublayer(streams, W, hc, fn):
    """streams [s, tokens, width] -> the new streams."""
    u = np.einsum("s,std->td", W[hc + "in"], streams)
    y = fn(u)
    return np.einsum("st,sxd->txd", W[hc + "mix"], streams) + W[hc + "out"][:, None, None] * y[None]


def sandwich_sublayer(x, W, p, n, eps, fn):
    """Norm before and after the sublayer, the result scaled channel by channel."""
    return x + W[f"{p}ls{n}"] * norm(fn(norm(x, W[f"{p}norm{n}"], eps)), W[f"{p}norm{n}b"], eps)


def forward_sandwich(tokens, cfg, W, dtype=np.float64, layers_out=None):
    """Logits [tokens, vocab] of a stack of sandwich sublayers in which every pass of the loop starts from a linear map of the
    residual row beside the embedding row."""
    W = {k: a.astype(dtype) for k, a in W.items()}
    eps = cfg["norm"]["eps"]
    x = x0 = W["embed"][np.asarray(tokens)]
    runs, loop = layer_runs(cfg), cfg.get("loop")
    for n, i in enumerate(runs):
        L, p = cfg["layers"][i], f"l{i}."
        if loop and loop["start"] <= n < loop["start"] + (loop["stop"] - loop["start"]) * loop["times"] and i == loop["start"]:
            x = np.concatenate([x, x0], axis=1) @ W["loop.in"].T
        x = sandwich_sublayer(x, W, p, 1, eps, lambda h: MIXERS[L["type"]](h, W, p + "mix.", L["mixer"], eps))
        if L.get("mlp"):
            x = sandwich_sublayer(x, W, p, 2, eps, lambda h: experts(h, W, p + "mlp.", L["mlp"]))
        if layers_out is not None:
            layers_out.append(x)
    return norm(x, W["final.norm"], eps) @ W["head"].T


def forward(tokens, cfg, W, dtype=np.float64, layers_out=None):
    """Logits [tokens, vocab] of one whole sequence; layers_out collects the sum of the streams after every layer run."""
    if cfg["architecture"] == "Zibovik":
        return forward_sandwich(tokens, cfg, W, dtype, layers_out)
    W = {k: a.astype(dtype) for k, a in W.items()}
    eps = cfg["norm"]["eps"]
    x = embed(np.asarray(tokens), W, cfg).astype(dtype)
    s = np.repeat(x[None], cfg.get("streams", 1), axis=0)
    for i in layer_runs(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        s = hyper_sublayer(s, W, p + "hc1.", lambda u: MIXERS[L["type"]](norm_around_zero(u, W[p + "norm1"], eps), W, p + "mix.", L["mixer"], eps))
        if L.get("mlp"):
            s = hyper_sublayer(s, W, p + "hc2.", lambda u: feed_forward(norm_around_zero(u, W[p + "norm2"], eps), W, p + "mlp."))
        if layers_out is not None:
            layers_out.append(s.sum(0))
    return norm_around_zero(s.sum(0), W["final.norm"], eps) @ W["head"].T
