"""Small configurations and random weights of block models for the tests, written as model directories."""
import json
import os

import numpy as np

import plain_blocks as P


def parallel_mixer(heads=4, kv_heads=2, dim=24, vdim=16, window=11, pool=4, left_scale=0.8, right_scale=0.5, scale=None, rheads=3, rdim=20, rvdim=12,
                   rot_dims=12, base=500.0, decay=None):
    return {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 1.3 * dim ** -0.5,
                     "mask": {"size": window, "pool": pool}},
            "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "decay": decay or [1 - 0.5 ** (i + 2) for i in range(rheads)],
                      "rot": {"base": base, "dims": rot_dims}},
            "left_scale": left_scale, "right_scale": right_scale}


def wkv_mixer(heads=3, dim=20):
    return {"heads": heads, "dim": dim}


def config(layers=("parallel", "wkv"), loop=None, vocab=301, width=88, ff=136, streams=3, buckets=53, mixer=None, wkv=None, mlp_none=(), eps=1e-5,
           embed_scale=2.5):
    ls = []
    for i, t in enumerate(layers):
        ls.append({"type": t, "mixer": parallel_mixer(**(mixer or {})) if t == "parallel" else wkv_mixer(**(wkv or {})),
                   "mlp": None if i in mlp_none else {"kind": "dense", "ff": ff}})
    return {"architecture": "Filulix", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
            "embedding": {"scale": embed_scale, "bigram": {"buckets": buckets, "mul_cur": 5, "mul_prev": 11}}, "layers": ls, "loop": loop}


def weights(cfg, seed=0, rank=7):
    """Random weights, rounded to bfloat16; matrices with unit gain, everything else away from the values that hide a fault."""
    rng = np.random.default_rng(seed)
    w, s, v = cfg["width"], cfg["streams"], cfg["vocab"]
    W = {}

    def mat(name, rows, cols, gain=1.0):
        W[name] = gain * rng.standard_normal((rows, cols)) / np.sqrt(cols)

    W["embed"] = rng.standard_normal((v, w))
    W["bigram"] = 1.5 * rng.standard_normal((cfg["embedding"]["bigram"]["buckets"] + 1, w))
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        for q in ("1", "2") if L["mlp"] else ("1",):
            W[p + "norm" + q] = 0.3 * rng.standard_normal(w)
            W[p + f"hc{q}.in"] = 0.5 + 0.5 * rng.random(s)
            W[p + f"hc{q}.out"] = 0.4 + rng.random(s)
            W[p + f"hc{q}.mix"] = 0.7 * np.eye(s) + 0.3 * rng.random((s, s)) / s
        if L["type"] == "parallel":
            a, b = m["left"], m["right"]
            mat(p + "mix.left.q", a["heads"] * a["dim"], w, 1.5)
            mat(p + "mix.left.k", a["kv_heads"] * a["dim"], w, 1.5)
            mat(p + "mix.left.v", a["kv_heads"] * a["vdim"], w)
            mat(p + "mix.left.o", w, a["heads"] * a["vdim"], 2.0)
            mat(p + "mix.right.q", b["heads"] * b["dim"], w)
            mat(p + "mix.right.k", b["heads"] * b["dim"], w)
            mat(p + "mix.right.v", b["heads"] * b["vdim"], w)
            mat(p + "mix.right.g", b["heads"] * b["vdim"], w)
            mat(p + "mix.right.o", w, b["heads"] * b["vdim"], 2.0)
        else:
            n = m["heads"] * m["dim"]
            for x in "rkvgw":
                W[p + "mix.mu." + x] = rng.random(w)
            for x in "rkvg":
                mat(p + "mix." + x, n, w)
            mat(p + "mix.w1", rank, w)
            mat(p + "mix.w2", n, rank)
            W[p + "mix.w0"] = -2.5 + 1.5 * rng.standard_normal(n)
            W[p + "mix.u"] = rng.standard_normal((m["heads"], m["dim"]))
            W[p + "mix.norm"] = 0.5 + rng.random(n)
            mat(p + "mix.o", w, n, 2.0)
        if L["mlp"]:
            mat(p + "mlp.gate", L["mlp"]["ff"], w)
            mat(p + "mlp.up", L["mlp"]["ff"], w)
            mat(p + "mlp.down", w, L["mlp"]["ff"], 2.0)
    W["final.norm"] = 0.3 * rng.standard_normal(w)
    mat("head", v, w)
    return {k: (P.to_bf16_bits(a).astype(np.uint32) << 16).view(np.float32).astype(np.float64) for k, a in W.items()}


def case(seed=0, **kw):
    cfg = config(**kw)
    return cfg, weights(cfg, seed)


# ------------------------------------------------------------------ latent attention and experts
def latent_mixer(heads=3, dim=20, rot_dim=6, vdim=12, kv_rank=28, window=11, base=700.0, scale=None, rot_dims=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window},
            "rot": {"base": base, "dims": rot_dims or rot_dim}, "scale": scale if scale is not None else 1.5 * (dim + rot_dim) ** -0.5}


def latent_config(layers=2, loop=None, vocab=211, width=88, mixer=None, mixers=None, experts=5, top=2, ff=24, mlp_none=(), eps=2e-5, moe=None):
    """mixers / moe: per-layer changes {layer: {...}} of the common mixer / (experts, top, ff)."""
    ls = []
    for i in range(layers):
        e = {"experts": experts, "top": top, "ff": ff, **((moe or {}).get(i, {}))}
        ls.append({"type": "latent_attention", "mixer": latent_mixer(**{**(mixer or {}), **((mixers or {}).get(i, {}))}),
                   "mlp": None if i in mlp_none else {"kind": "moe", "expert": {"ff": e["ff"]}, "router": {"experts": e["experts"], "top": e["top"]}}})
    cfg = {"architecture": "Zibovik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": ls}
    if loop:
        cfg["loop"] = loop
    return cfg


def latent_weights(cfg, seed=0, clear_routing=True):
    """Random weights, rounded to bfloat16.  clear_routing: the last channels of the residual hold values that only the
    embedding writes, a few well separated levels per token, and the routers read nothing else - the choice of experts is never
    close, whatever rounding does to a row."""
    rng = np.random.default_rng(seed)
    w, v = cfg["width"], cfg["vocab"]
    W = {}

    def mat(name, rows, cols, gain=1.0):
        W[name] = gain * rng.standard_normal((rows, cols)) / np.sqrt(cols)

    most = max([L["mlp"]["router"]["experts"] for L in cfg["layers"] if L["mlp"]], default=0) if clear_routing else 0
    assert most < w
    free = w - most  # channels sublayers may write
    W["embed"] = rng.standard_normal((v, w))
    for t in range(v if most else 0):
        W["embed"][t, free:] = rng.permutation(np.linspace(-2.0, 2.0, most) if most > 1 else [1.0])
    if cfg.get("loop"):
        mat("loop.in", w, 2 * w, 1.2)
        W["loop.in"][free:] = 0
        for c in range(free, w):
            W["loop.in"][c, c], W["loop.in"][c, w + c] = 0.75, 0.25
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        H, D, R, DV, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        for n in "12" if L["mlp"] else "1":
            W[p + "norm" + n] = 0.5 + rng.random(w)
            W[p + f"norm{n}b"] = 0.5 + rng.random(w)
            W[p + "ls" + n] = 0.3 + rng.random(w)
        mat(p + "mix.q", H * (D + R), w)
        mat(p + "mix.dkv", C + R, w)
        W[p + "mix.dkv.norm"] = 0.5 + rng.random(C)
        mat(p + "mix.uk", H * D, C)
        mat(p + "mix.uv", H * DV, C)
        W[p + "mix.sink"] = 1.5 + rng.standard_normal(H)
        mat(p + "mix.g", H, w, 1.5)
        mat(p + "mix.o", w, H * DV, 2.0)
        W[p + "mix.o"][free:] = 0
        if L["mlp"]:
            E, ff = L["mlp"]["router"]["experts"], L["mlp"]["expert"]["ff"]
            for e in range(E):
                mat(p + f"mlp.e{e}.gate", ff, w, 1.5)
                mat(p + f"mlp.e{e}.up", ff, w, 1.5)
                mat(p + f"mlp.e{e}.down", w, ff, 2.0)
                W[p + f"mlp.e{e}.down"][free:] = 0
            mat(p + "mlp.router", E, w, 2.0)
            if most:
                W[p + "mlp.router"][:] = 0
                W[p + "norm2"][free:] = 1.0
                for e in range(E):
                    W[p + "mlp.router"][e, free + e] = 1.5
    W["final.norm"] = 0.5 + rng.random(w)
    mat("head", v, w)
    return {k: (P.to_bf16_bits(a).astype(np.uint32) << 16).view(np.float32).astype(np.float64) for k, a in W.items()}


def latent_case(seed=0, clear_routing=True, **kw):
    cfg = latent_config(**kw)
    return cfg, latent_weights(cfg, seed, clear_routing)


def write(path, cfg, W):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    P.write_safetensors(os.path.join(path, "model.safetensors"), W)
    return str(path)


def tokens(cfg, n, seed=0):
    return np.random.default_rng(1000 + seed).integers(0, cfg["vocab"], n).tolist()
