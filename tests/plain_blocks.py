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


MIXERS = {"parallel": parallel, "wkv": wkv}


def feed_forward(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


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


def forward(tokens, cfg, W, dtype=np.float64, layers_out=None):
    """Logits [tokens, vocab] of one whole sequence; layers_out collects the sum of the streams after every layer run."""
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
