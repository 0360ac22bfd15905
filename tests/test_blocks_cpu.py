"""Block models, host side: the configuration reader and registry through the C ABI, and the plain implementation's own
invariants (what the GPU tests compare against has to be right on its own)."""
import copy

import numpy as np
import pytest

import block_cases as B
import plain_blocks as P


def test_registry_names_the_architecture(lcu):
    assert "Filulix" in lcu.architectures()


@pytest.mark.parametrize("loop,n,want", [(None, 3, [0, 1, 2]), ({"start": 0, "stop": 3, "times": 2}, 3, [0, 1, 2] * 2),
                                         ({"start": 1, "stop": 2, "times": 4}, 3, [0, 1, 1, 1, 1, 2]),
                                         ({"start": 1, "stop": 3, "times": 1}, 4, [0, 1, 2, 3]), ({"start": 2, "stop": 2, "times": 5}, 3, [0, 1, 2])])
def test_layer_runs(lcu, loop, n, want):
    cfg = B.config(layers=["parallel", "wkv", "parallel", "wkv"][:n], loop=loop)
    assert lcu.config_runs(cfg) == want == P.layer_runs(cfg)


def test_bad_configurations_are_named(lcu):
    good = B.config()
    lcu.config_runs(good)
    for change, text in [((lambda c: c.update(architecture="Nothing")), "not known"), ((lambda c: c.pop("width")), "width"),
                         ((lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=5)), "multiple"),
                         ((lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5])), "decays"),
                         ((lambda c: c["layers"][0].update(type="other")), "other"),
                         ((lambda c: c["layers"][0].update(mlp={"kind": "sparse", "ff": 8})), "sparse"),
                         ((lambda c: c.update(loop={"start": 0, "stop": 9, "times": 2})), "loop")]:
        bad = copy.deepcopy(good)
        change(bad)
        with pytest.raises(lcu.LcuError, match=text):
            lcu.config_runs(bad)


def test_malformed_text_is_an_error(lcu):
    for text in (b"", b"{", b'{"architecture": }', b"[1, 2"):
        assert lcu.lib.lcu_config_runs(text, lcu._ptr(np.empty(8, np.int32)), 8) < 0


# ------------------------------------------------------------------ the plain implementation
def test_plain_forward_is_causal():
    cfg, W = B.case(seed=3, layers=["parallel", "wkv"], loop={"start": 0, "stop": 2, "times": 2})
    t = B.tokens(cfg, 40, 1)
    a = P.forward(t, cfg, W)
    b = P.forward(t[:25], cfg, W)
    assert np.abs(a[:25] - b).max() < 1e-9


def test_plain_window_edges():
    """What a position sees, from the definition: tokens i - size + 1 .. i and the blocks that end at i - size or before."""
    m = {"heads": 1, "kv_heads": 1, "dim": 4, "vdim": 4, "scale": 0.0, "mask": {"size": 5, "pool": 3}}
    T = 20
    h = np.eye(T)
    W = {"q": np.zeros((4, T)), "k": np.zeros((4, T)), "v": np.zeros((4, T)), "o": np.eye(4)}
    for j in range(T):  # value of token j counts it; equal scores: the output is the share of keys that hold it
        W["v"][:] = 0
        W["v"][0, j] = 1
        o = P.window_pool_attention(h, W, "", m)[:, 0]
        for i in range(T):
            blocks = [b for b in range(T // 3) if 3 * b + 2 <= i - 5]
            keys = len(blocks) + min(i + 1, 5)
            want = 1 / keys if max(0, i - 4) <= j <= i else (1 / 3 / keys if j // 3 in blocks else 0.0)
            assert abs(o[i] - want) < 1e-12, (i, j)


def test_plain_recurrences_against_their_closed_forms():
    rng = np.random.default_rng(5)
    T, D = 12, 6
    h = rng.standard_normal((T, D))
    m = {"heads": 1, "dim": D, "vdim": D, "decay": [0.7]}
    W = {n: rng.standard_normal((D, D)) for n in "qkvo"} | {"g": np.zeros((D, D))}
    W["g"][:] = 1e3 * np.eye(D)  # (silu is the identity or zero here; only positive gates are compared)
    q, k, v = (h @ W[n].T for n in "qkv")
    A = np.tril(q @ k.T * D ** -0.5 * 0.7 ** (np.arange(T)[:, None] - np.arange(T)[None]))
    want = P.unit_rms(A @ v, 1e-6) * P.silu(h @ W["g"].T) @ W["o"].T
    assert np.allclose(P.retention(h, W, "", m, 1e-6), want)


def test_plain_hyper_connections_with_one_plain_stream_are_a_residual_sum():
    x = np.random.default_rng(1).standard_normal((1, 5, 3))
    W = {"in": np.ones(1), "out": np.ones(1), "mix": np.ones((1, 1))}
    assert np.allclose(P.hyper_sublayer(x, W, "", lambda u: 2 * u), 3 * x)


def test_safetensors_round_trip(tmp_path):
    a = {"x": np.arange(6, dtype=np.float64).reshape(2, 3) / 4, "y": np.array([1.0, -2.5])}
    P.write_safetensors(tmp_path / "f", a)
    b = P.read_safetensors(tmp_path / "f")
    assert all(np.array_equal(a[n], b[n]) for n in a)
