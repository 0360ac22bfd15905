"""Latent attention, routed feed-forward and their stack, host side: the configuration reader through the C ABI, the plain
implementation's mechanisms against closed forms, and that the mistakes the GPU tests are meant to catch would show."""
import copy

import numpy as np
import pytest

import block_cases as B
import plain_blocks as P


def test_registry_names_the_architecture(lcu):
    assert "Zibovik" in lcu.architectures()


@pytest.mark.parametrize("loop,n,want", [(None, 3, [0, 1, 2]), ({"start": 0, "stop": 3, "times": 2}, 3, [0, 1, 2] * 2),
                                         ({"start": 1, "stop": 2, "times": 4}, 3, [0, 1, 1, 1, 1, 2]), ({"start": 1, "stop": 3, "times": 1}, 4, [0, 1, 2, 3])])
def test_layer_runs(lcu, loop, n, want):
    cfg = B.latent_config(layers=n, loop=loop)
    assert lcu.config_runs(cfg) == want == P.layer_runs(cfg)


def test_bad_configurations_are_named(lcu):
    good = B.latent_config()
    lcu.config_runs(good)
    mixer = lambda c: c["layers"][0]["mixer"]  # noqa: E731
    router = lambda c: c["layers"][1]["mlp"]["router"]  # noqa: E731
    for change, text in [((lambda c: mixer(c).pop("kv_rank")), "kv_rank"), ((lambda c: mixer(c).pop("rot")), "rot"), ((lambda c: mixer(c).pop("mask")), "mask"),
                         ((lambda c: mixer(c)["rot"].update(dims=8)), "rotated"), ((lambda c: mixer(c)["rot"].update(dims=3)), "rotated"),
                         ((lambda c: mixer(c).update(kv_rank=5000)), "latent"), ((lambda c: router(c).update(top=6)), "top 6 of 5"),
                         ((lambda c: router(c).update(experts=0)), "experts"), ((lambda c: c["layers"][0].update(type="wkv")), "wkv"),
                         ((lambda c: c["layers"][1]["mlp"].pop("expert")), "expert"), ((lambda c: c["norm"].pop("eps")), "eps")]:
        bad = copy.deepcopy(good)
        change(bad)
        with pytest.raises(lcu.LcuError, match=text):
            lcu.config_runs(bad)


# ------------------------------------------------------------------ the plain implementation
def test_plain_rotation_is_a_complex_product():
    rng = np.random.default_rng(0)
    x, pos = rng.standard_normal((9, 2, 10)), np.arange(9) * 3.0
    got = P.rotate_pairs(x, pos, 100.0, 6)
    z = (x[..., 0:6:2] + 1j * x[..., 1:6:2]) * np.exp(1j * pos[:, None, None] * 100.0 ** (-np.arange(3) / 3.0))
    assert np.allclose(got[..., 0:6:2], z.real) and np.allclose(got[..., 1:6:2], z.imag) and np.array_equal(got[..., 6:], x[..., 6:])


def test_plain_window_and_sink():
    """Equal scores of zero: every visible key has the share 1 / (keys + exp(sink))."""
    T, size = 14, 5
    q, v = np.zeros((T, 1, 3)), np.eye(T)[:, None, :]
    for sink in (None, np.array([0.7])):
        o = P.window_softmax(q, q, v, 1.0, size, sink)[:, 0]
        for i in range(T):
            seen = [j for j in range(T) if 0 <= i - j < size]
            share = 1 / (len(seen) + (0 if sink is None else np.exp(0.7)))
            assert np.allclose(o[i], [share if j in seen else 0.0 for j in range(T)])


def test_plain_latent_attention_is_attention_on_cache_rows():
    """Scores and results formed from latents directly (queries through the key matrix, results through the value matrix)."""
    cfg, W = B.latent_case(seed=4, layers=1)
    m, p, eps = cfg["layers"][0]["mixer"], "l0.mix.", cfg["norm"]["eps"]
    H, D, R, DV, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = 17
    h = np.random.default_rng(1).standard_normal((T, cfg["width"]))
    pos = np.arange(T) * 1.0
    q = (h @ W[p + "q"].T).reshape(T, H, D + R)
    d = h @ W[p + "dkv"].T
    c = P.norm(d[:, :C], W[p + "dkv.norm"], eps)
    row = np.concatenate([c, P.rotate_pairs(d[:, None, C:], pos, m["rot"]["base"], R)[:, 0]], axis=1)
    uk, uv = W[p + "uk"].reshape(H, D, C), W[p + "uv"].reshape(H, DV, C)
    out = np.zeros((T, H, DV))
    for hd in range(H):
        qa = np.concatenate([q[:, hd, :D] @ uk[hd], P.rotate_pairs(q[:, hd:hd + 1, D:], pos, m["rot"]["base"], R)[:, 0]], axis=1)
        s = qa @ row.T * m["scale"]
        i, j = np.arange(T)[:, None], np.arange(T)[None]
        e = np.where((i >= j) & (i - j < m["mask"]["size"]), np.exp(s), 0)
        a = e / (e.sum(1, keepdims=True) + np.exp(W[p + "sink"][hd]))
        out[:, hd] = a @ c @ uv[hd].T * P.sigmoid(h @ W[p + "g"][hd])[:, None]
    assert np.allclose(P.latent_attention(h, W, p, m, eps), out.reshape(T, -1) @ W[p + "o"].T)


def test_plain_experts():
    """All experts chosen: a plain sum; the weights are the scores as they are, on the expert's input."""
    cfg, W = B.latent_case(seed=5, layers=1, experts=3, top=3, clear_routing=False)
    h = np.random.default_rng(2).standard_normal((4, cfg["width"]))
    s = P.sigmoid(h @ W["l0.mlp.router"].T)
    want = sum(P.feed_forward(s[:, e:e + 1] * h, W, f"l0.mlp.e{e}.") for e in range(3))
    assert np.allclose(P.experts(h, W, "l0.mlp.", cfg["layers"][0]["mlp"]), want)
    cfg["layers"][0]["mlp"]["router"]["top"] = 1
    best = s.argmax(1)
    one = P.experts(h, W, "l0.mlp.", cfg["layers"][0]["mlp"])
    for t in range(4):
        assert np.allclose(one[t], P.feed_forward(s[t, best[t]] * h[t:t + 1], W, f"l0.mlp.e{best[t]}.")[0])


def test_plain_forward_is_causal():
    cfg, W = B.latent_case(seed=3, layers=3, loop={"start": 0, "stop": 2, "times": 2})
    t = B.tokens(cfg, 40, 1)
    assert np.abs(P.forward(t, cfg, W)[:25] - P.forward(t[:25], cfg, W)).max() < 1e-9


def mistakes():
    """What a wrong implementation of one mechanism computes, as patches of the plain one."""
    def softmax(**change):
        f = P.window_softmax

        def g(q, k, v, scale, size, sink=None):
            a = dict(scale=scale, size=size, sink=sink)
            a.update({n: c(a) for n, c in change.items()})
            return f(q, k, v, **a)
        return "window_softmax", g

    def half(x, positions, base, dims):
        out, n = x.copy(), dims // 2
        perm = [i // 2 + (i % 2) * n for i in range(dims)]
        y = np.empty_like(x[..., :dims])
        y[..., list(range(dims))] = x[..., perm]
        y = rotate(y, positions, base, dims)
        out[..., perm] = y
        return out

    rotate, norm, feed, route = P.rotate_pairs, P.norm, P.feed_forward, P.route

    def renormalised(h, W, p, top):
        pick, w = route(h, W, p, top)
        return pick, w / w.sum(1, keepdims=True)

    def output_weighted(h, W, p, m):
        pick, weight = route(h, W, p, m["router"]["top"])
        return np.stack([sum(w * feed(h[t:t + 1], W, f"{p}e{e}.")[0] for e, w in zip(pick[t], weight[t])) for t in range(len(h))])

    return {"no sink": softmax(sink=lambda a: None), "sink scaled": softmax(sink=lambda a: a["sink"] * a["scale"]),
            "window one longer": softmax(size=lambda a: a["size"] + 1), "window one shorter": softmax(size=lambda a: a["size"] - 1),
            "rotation of halves": ("rotate_pairs", half), "rotation backwards": ("rotate_pairs", lambda x, p, b, d: rotate(x, -p, b, d)),
            "one position off": ("rotate_pairs", lambda x, p, b, d: rotate(x, p + (x.shape[1] == 1), b, d)),
            "norms around zero": ("norm", lambda x, w, eps: norm(x, 1 + w, eps)), "weights renormalised": ("route", renormalised),
            "one expert fewer": ("route", lambda h, W, p, top: route(h, W, p, top - 1)), "weight on the output": ("experts", output_weighted)}


@pytest.mark.parametrize("name", sorted(mistakes()))
def test_mistakes_would_show(monkeypatch, name):
    cfg, W = B.latent_case(seed=7, layers=2, loop={"start": 0, "stop": 1, "times": 2})
    t = B.tokens(cfg, 40, 2)
    want = P.forward(t, cfg, W)
    attr, wrong = mistakes()[name]
    monkeypatch.setattr(P, attr, wrong)
    d = P.forward(t, cfg, W) - want
    assert np.sqrt((d * d).mean(1)).max() / np.sqrt((want * want).mean()) > 0.12  # (three times the bfloat16 limit)


@pytest.mark.parametrize("name", ["ls1", "ls2", "norm1b", "norm2b", "mix.g", "mix.dkv.norm"])
def test_missing_factors_would_show(name):
    cfg, W = B.latent_case(seed=8, layers=1)
    t = B.tokens(cfg, 30, 2)
    want = P.forward(t, cfg, W)
    W["l0." + name] = np.zeros_like(W["l0." + name]) if name == "mix.g" else np.ones_like(W["l0." + name])
    d = P.forward(t, cfg, W) - want
    assert np.sqrt((d * d).mean(1)).max() / np.sqrt((want * want).mean()) > 0.12
