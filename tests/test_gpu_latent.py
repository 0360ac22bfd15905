"""Zibovik on the GPU against the plain implementation: latent attention, sink and gates, experts, sandwich norms and looped
passes alone and stacked, in both number formats; prompts against token-by-token decoding, portions, reuse of a context,
window edges, long decoding, other kernels for the same work, greedy generation, the replay program."""
import copy
import json
import os
import subprocess

import numpy as np
import pytest

import block_cases as B
import plain_blocks as P
from block_runs import DTYPES, LIMIT, WHOLE, both, check, row_errors, run  # noqa: F401 (run: fixture)

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

CASES = {
    "attention": dict(layers=1, mlp_none=(0,)),
    "attention, one head": dict(layers=1, mlp_none=(0,), mixer=dict(heads=1, dim=9, rot_dim=2, vdim=5, kv_rank=7)),
    "attention, nothing padded": dict(layers=1, mlp_none=(0,), width=256, mixer=dict(heads=4, dim=48, rot_dim=16, vdim=64, kv_rank=256, window=30)),
    "attention, 128 columns": dict(layers=1, mlp_none=(0,), mixer=dict(heads=2, dim=100, rot_dim=28, vdim=96, kv_rank=40)),
    "attention, 192 columns": dict(layers=1, mlp_none=(0,), mixer=dict(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=512)),
    "attention, 256 columns": dict(layers=1, mlp_none=(0,), mixer=dict(heads=2, dim=190, rot_dim=62, vdim=33, kv_rank=100)),
    "attention, more columns": dict(layers=1, mlp_none=(0,), mixer=dict(heads=2, dim=200, rot_dim=72, vdim=40, kv_rank=60)),
    "attention, wide values": dict(layers=1, mlp_none=(0,), mixer=dict(heads=2, dim=12, rot_dim=10, vdim=150, kv_rank=90)),
    "attention, small latent": dict(layers=1, mlp_none=(0,), mixer=dict(heads=5, kv_rank=3)),
    "attention, large latent": dict(layers=1, mlp_none=(0,), mixer=dict(heads=2, kv_rank=700)),
    "attention, many heads": dict(layers=1, mlp_none=(0,), mixer=dict(heads=19, dim=8, rot_dim=8, vdim=8, kv_rank=33)),
    "attention, window of one": dict(layers=1, mlp_none=(0,), mixer=dict(window=1)),
    "attention, window beyond the sequence": dict(layers=1, mlp_none=(0,), mixer=dict(window=100000)),
    "attention, part of the shared key turns": dict(layers=1, mlp_none=(0,), mixer=dict(rot_dim=12, rot_dims=8)),
    "one expert of five": dict(layers=1, top=1),
    "the only expert": dict(layers=1, experts=1, top=1, ff=40),
    "all experts": dict(layers=1, experts=4, top=4),
    "three of thirteen": dict(layers=1, experts=13, top=3, ff=17),
    "eleven of forty": dict(layers=1, experts=40, top=11, ff=9),
    "wide experts": dict(layers=1, experts=3, top=2, ff=300),
    "odd width": dict(layers=2, width=75, vocab=97),
    "loop from the start": dict(layers=3, loop={"start": 0, "stop": 2, "times": 2}),
    "loop in the middle": dict(layers=3, loop={"start": 1, "stop": 2, "times": 3}, mlp_none=(1,)),
    "loop over the end": dict(layers=2, loop={"start": 1, "stop": 2, "times": 2}, vocab=1003),
    "loop of one pass": dict(layers=2, loop={"start": 0, "stop": 2, "times": 1}),
    "unequal layers": dict(layers=3, mixers={0: dict(heads=2, dim=16, window=40), 2: dict(heads=4, vdim=21, kv_rank=50, window=5, base=90.0)},
                           moe={1: dict(experts=3, top=1, ff=50), 2: dict(experts=7, top=4)}, mlp_none=(0,)),
    "wider": dict(layers=2, width=384, experts=6, top=2, ff=128, mixer=dict(heads=6, dim=64, rot_dim=32, vdim=64, kv_rank=192, window=40)),
}


@both
@pytest.mark.parametrize("name", sorted(CASES))
def test_against_plain_whole_and_token_by_token(run, name, dtype):  # noqa: F811
    # (a seed whose only head is nowhere close to zero: the output norm would amplify bfloat16 rounding)
    cfg, W = B.latent_case(seed=4 if name == "attention, one head" else len(name), **CASES[name])
    t = B.tokens(cfg, 75, len(name))
    want = P.forward(t, cfg, W)
    r = run(cfg, W, dtype)
    check(r.feed(t, WHOLE), want, dtype)
    check(r.feed(t, [1]), want, dtype)  # every token through the captured step
    check(r.feed(t, [30, 1]), want, dtype)


def test_routing_on_everything_a_row_holds(run):  # noqa: F811
    """Routers that read the whole row, where the choice of experts is as close as it comes (binary32)."""
    cfg, W = B.latent_case(seed=31, clear_routing=False, layers=2, experts=9, top=3)
    t = B.tokens(cfg, 120, 5)
    r = run(cfg, W, "float32")
    want = P.forward(t, cfg, W)
    check(r.feed(t, WHOLE), want, "float32")
    check(r.feed(t, [50, 1]), want, "float32")


@both
@pytest.mark.parametrize("cuts", [[2], [3, 2, 7], [16], [17, 1, 1, 2], [64, 2], [5, 1, 30]])
def test_portions(run, cuts, dtype):  # noqa: F811
    cfg, W = B.latent_case(seed=9, layers=3, loop={"start": 0, "stop": 2, "times": 2}, mixers={2: dict(window=23)})
    t = B.tokens(cfg, 90, 3)
    check(run(cfg, W, dtype).feed(t, cuts), P.forward(t, cfg, W), dtype)


@both
def test_context_is_reused_by_the_next_sequence(run, dtype):  # noqa: F811
    cfg, W = B.latent_case(seed=4)
    r = run(cfg, W, dtype)
    for i, (n, cuts) in enumerate([(80, WHOLE), (1, [1]), (33, [2]), (70, [1]), (5, WHOLE), (2, [1])]):
        t = B.tokens(cfg, n, 20 + i)
        check(r.feed(t, cuts), P.forward(t, cfg, W), dtype)


@both
def test_contexts_beside_each_other(lcu, run, dtype):  # noqa: F811
    """Two requests of unequal length on contexts of their own, step by step in turn: each as if it were alone."""
    cfg, W = B.latent_case(seed=41, loop={"start": 0, "stop": 1, "times": 2})
    r = run(cfg, W, dtype)
    other = lcu.Context(r.model, context_len=128, temperature=1.0)
    try:
        for ctx, toks in ((r.ctx, B.tokens(cfg, 60, 1)), (other, B.tokens(cfg, 25, 2))):
            ctx.clear_tokens()
            ctx.plan = (toks, P.forward(toks, cfg, W))
        cuts = [7, 1, 2, 1, 9, 1]
        at = {id(r.ctx): 0, id(other): 0}
        for i in range(40):
            for ctx in (r.ctx, other):
                toks, want = ctx.plan
                a = at[id(ctx)]
                b = min(len(toks), a + cuts[i % len(cuts)])
                if b > a:
                    check(ctx.step(toks[a:b], list(range(b - a))), want[a:b], dtype, factor=1.5)  # (shares of few rows' own RMS)
                at[id(ctx)] = b
    finally:
        other.close()


@both
def test_first_tokens(run, dtype):  # noqa: F811
    cfg, W = B.latent_case(seed=6, loop={"start": 0, "stop": 1, "times": 2})
    r = run(cfg, W, dtype)
    for n in (1, 2, 3, 4):
        t = B.tokens(cfg, n, n)
        want = P.forward(t, cfg, W)
        check(r.feed(t, WHOLE), want, dtype)
        check(r.feed(t, [1]), want, dtype)


def standout_case(window, seed=2):
    """One attention layer in which token 0's key dwarfs all others for every query: whoever sees it shows it."""
    cfg, W = B.latent_case(seed=seed, layers=1, mlp_none=(0,), width=96, mixer=dict(window=window, heads=2, dim=16, rot_dim=8, vdim=16, kv_rank=24, scale=0.2))
    W["embed"][:, 0], W["embed"][:, 1] = 3.0, 0.0   # channel 0: the same in every token, channel 1: token 0 only
    W["embed"][0, 1] = 8.0
    W["l0.norm1"][:] = 1
    W["l0.mix.dkv.norm"][:] = 1
    W["l0.mix.q"][:] = 0
    W["l0.mix.q"][::24, 0] = 4.0                    # first unrotated query dimension of both heads
    W["l0.mix.dkv"][0] = 0
    W["l0.mix.dkv"][0, 1] = 3.0                     # latent 0 is token 0's alone
    W["l0.mix.uk"][:] = 0
    W["l0.mix.uk"][::16, 0] = 2.0
    W["l0.mix.sink"][:] = 2.0
    return cfg, W


@both
@pytest.mark.parametrize("window", [13, 64, 65, 130])
def test_window_edges(run, window, dtype):  # noqa: F811
    cfg, W = standout_case(window)
    n = 2 * window + 20
    r = run(cfg, W, dtype, context_len=512)
    for at in (0, 1, 7, window - 1, window):
        t = [1 + x % (cfg["vocab"] - 1) for x in B.tokens(cfg, n, at)]
        t[at] = 0
        want = P.forward(t, cfg, W)
        for d in (-1, 1):  # a window one off is far outside the limit somewhere
            c = copy.deepcopy(cfg)
            c["layers"][0]["mixer"]["mask"]["size"] += d
            assert row_errors(P.forward(t, c, W), want).max() > 3 * LIMIT["bfloat16"]
        for cuts in (WHOLE, [1], [window, 1], [at + 1, 2], [window - 1, 3]):
            check(r.feed(t, cuts), want, dtype)


@both
def test_far_key(run, dtype):  # noqa: F811
    """A key hundreds of positions back is seen by a wide window, and its loss would show."""
    cfg, W = standout_case(600)
    t = [1 + x % (cfg["vocab"] - 1) for x in B.tokens(cfg, 420, 5)]
    t[9] = 0
    want = P.forward(t, cfg, W)
    gone = list(t)
    gone[9] = 1
    assert row_errors(P.forward(gone, cfg, W)[-3:], want[-3:]).min() > 3 * LIMIT["bfloat16"]
    r = run(cfg, W, dtype, context_len=512)
    check(r.feed(t, WHOLE), want, dtype)
    check(r.feed(t, [400, 1]), want, dtype)


@both
@pytest.mark.parametrize("sink", [-30.0, 9.0, 60.0])
def test_extreme_sinks(run, sink, dtype):  # noqa: F811
    """Sinks far below and far above every score: no overflow, the shares stay right."""
    cfg, W = B.latent_case(seed=21, layers=1, mlp_none=(0,))
    W["l0.mix.sink"][:] = sink
    W["l0.norm1b"][:] = 1
    t = B.tokens(cfg, 40, 3)
    if sink > 10:  # (what is left of the heads is below the norm's eps: the sublayer adds nothing)
        cfg["norm"]["eps"] = 1e-3
    want = P.forward(t, cfg, W)
    r = run(cfg, W, dtype)
    check(r.feed(t, WHOLE), want, dtype)
    check(r.feed(t, [1]), want, dtype)


@both
def test_long_decoding(run, dtype):  # noqa: F811
    cfg, W = B.latent_case(seed=8, mixer=dict(window=24))
    t = B.tokens(cfg, 420, 7)
    check(run(cfg, W, dtype, context_len=430).feed(t, [4, 1]), P.forward(t, cfg, W), dtype)


def test_passes_longer_than_the_row_buffers(run):  # noqa: F811
    cfg, W = B.latent_case(seed=12, layers=2, width=64, vocab=64, experts=4, top=2, ff=24, loop={"start": 0, "stop": 1, "times": 2},
                           mixer=dict(heads=2, dim=16, rot_dim=8, vdim=24, kv_rank=32, window=100))
    t = B.tokens(cfg, 2500, 2)
    want = P.forward(t, cfg, W)
    for dtype in DTYPES:
        r = run(cfg, W, dtype, context_len=2600)
        check(r.feed(t, WHOLE), want, dtype)


@pytest.mark.parametrize("width", [256, 384])
@pytest.mark.parametrize("keys", [{}, {"prefill_group_tile": 128}, {"prefill_group_tile": 256}, {"block_attn_mma": 0}, {"use_graph": 0, "use_pdl": 0},
                                  {"prompt_pdl": 0}, {"block_row_one_cta": 0}])
def test_kernel_choices_agree(lcu, run, keys, width):  # noqa: F811
    """Other kernels for the same products and attention: 128- and 256-row tiles of the experts' products, the per-row
    attention, steps without a graph, launches one after the other, a single row on a cluster."""
    defaults = {"prefill_group_tile": 0, "block_attn_mma": 1, "use_graph": 1, "use_pdl": 1, "prompt_pdl": 1, "block_row_one_cta": 2048}
    cfg, W = B.latent_case(seed=14, layers=2, width=width, experts=3, top=2, ff=320, mixer=dict(heads=4, dim=64, rot_dim=32, vdim=64, kv_rank=128, window=48))
    t = B.tokens(cfg, 600, 4)
    want = P.forward(t, cfg, W)
    try:
        for k, v in keys.items():
            lcu.check(lcu.lib.lcu_set_tuning(k.encode(), v))
        check(run(cfg, W, "bfloat16", context_len=640).feed(t, [590, 1]), want, "bfloat16")
    finally:
        for k in keys:
            lcu.check(lcu.lib.lcu_set_tuning(k.encode(), defaults[k]))


def test_one_expert_takes_every_row(run):  # noqa: F811
    """All tokens to the same experts: some row groups are full tiles, the others empty."""
    cfg, W = B.latent_case(seed=15, layers=1, experts=6, top=2)
    free = cfg["width"] - 6
    W["embed"][:, free:] = [2.0, -1.0, 1.0, -2.0, 0.0, -1.5]
    t = B.tokens(cfg, 400, 4)
    want = P.forward(t, cfg, W)
    for dtype in DTYPES:
        check(run(cfg, W, dtype, context_len=512).feed(t, [395, 1]), want, dtype)


def greedy(cfg, W, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(P.forward(seq, cfg, W)[-1].argmax()))
    return seq[len(prompt):]


def test_greedy_generation(run):  # noqa: F811
    """next_token and the device-chained loop pick the plain implementation's argmax, token after token."""
    cfg, W = B.latent_case(seed=16, layers=2, loop={"start": 0, "stop": 1, "times": 2})
    r = run(cfg, W, "float32")
    prompt = B.tokens(cfg, 12, 9)
    want = greedy(cfg, W, prompt, 16)
    r.ctx.clear_tokens()
    got = [r.ctx.next_token(prompt)]
    while len(got) < 16:
        got.append(r.ctx.next_token([got[-1]]))
    assert got == want
    r.ctx.clear_tokens()
    first = r.ctx.next_token(prompt)
    toks, ms = r.ctx.decode_chained(first, 15)
    assert [first] + toks.tolist() == want and ms > 0
    assert r.ctx.tokens_left() == 256 - len(prompt) - 15


def test_greedy_generation_in_bfloat16(run):  # noqa: F811
    """Every generated token is the plain implementation's choice, or as good as its choice within the rounding of a row."""
    cfg, W = B.latent_case(seed=17, layers=2)
    r = run(cfg, W, "bfloat16")
    prompt = B.tokens(cfg, 20, 9)
    r.ctx.clear_tokens()
    first = r.ctx.next_token(prompt)
    toks, _ = r.ctx.decode_chained(first, 30)
    seq = prompt + [first] + toks.tolist()
    lg = P.forward(seq, cfg, W)
    for i in range(len(prompt), len(seq)):
        row = lg[i - 1]
        assert row.max() - row[seq[i]] < 4 * LIMIT["bfloat16"] * np.sqrt((row * row).mean()), i


def test_sampling_repeats_for_a_seed(run):  # noqa: F811
    cfg, W = B.latent_case(seed=18)
    W["head"] *= 0.2
    r = run(cfg, W, "bfloat16")
    seen = []
    for seed in (5, 5, 6):
        r.ctx.clear_tokens()
        r.ctx.set_sampling(1, seed)
        t = r.ctx.next_token(B.tokens(cfg, 6, 3))
        seen.append([t] + r.ctx.decode_chained(t, 20)[0].tolist())
    assert seen[0] == seen[1] != seen[2]


def test_errors(lcu, run, tmp_path):  # noqa: F811
    cfg, W = B.latent_case(seed=19, loop={"start": 0, "stop": 1, "times": 2})
    r = run(cfg, W, "bfloat16", context_len=16)
    with pytest.raises(lcu.LcuError, match="context length"):
        r.ctx.step(B.tokens(cfg, 17))
    assert r.model.family() == "Zibovik"
    for name in ("l1.mix.sink", "loop.in", "l0.mlp.e3.up", "l1.norm2b", "l0.ls1"):
        gone = dict(W)
        gone.pop(name)
        with pytest.raises(lcu.LcuError, match=name.replace(".", r"\.")):
            lcu.Model.load(B.write(tmp_path / name, cfg, gone))
    with pytest.raises(lcu.LcuError, match="mix.uk"):
        lcu.Model.load(B.write(tmp_path / "shape", cfg, dict(W, **{"l0.mix.uk": W["l0.mix.uk"][:, :-1]})))


@both
def test_replay_program(tmp_path, dtype):
    cfg, W = B.latent_case(seed=20, layers=2, loop={"start": 1, "stop": 2, "times": 2})
    path = B.write(tmp_path / "m", cfg, W)
    out = tmp_path / "out"
    out.mkdir()
    seqs = {"x": B.tokens(cfg, 50, 1), "y": B.tokens(cfg, 7, 2)}
    steps, want = [], []
    for rid, cuts in (("x", [40, 2, 1, 1, 6]), ("y", [1, 1, 5])):
        at = 0
        full = P.forward(seqs[rid], cfg, W)
        for n in cuts:
            w = [] if n == 2 else [0, n - 1]
            steps.append({"step": len(steps), "entries": [{"id": rid, "tokens": seqs[rid][at:at + n], "want": w}],
                          "end": [rid] if at + n == len(seqs[rid]) else []})
            want.append(full[[at + i for i in w]])
            at += n
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(out), "--max-tokens", "64"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done ")] == [f"done {i}" for i in range(len(steps))]
    for i, w in enumerate(want):
        f = out / f"{i}.f32"
        assert f.exists() == bool(len(w))
        if len(w):
            check(np.fromfile(f, np.float32).reshape(len(w), cfg["vocab"]), w, dtype, factor=1.5)


@both
def test_many_chunks_of_keys(run, dtype):  # noqa: F811
    """A window of more rows than a decode step's buffers hold at once, also with long cache rows."""
    for mixer in (dict(heads=2, window=3000, kv_rank=48), dict(heads=1, window=1200, kv_rank=700)):
        cfg, W = B.latent_case(seed=33, layers=1, mlp_none=(0,), mixer=mixer)
        t = B.tokens(cfg, 1400, 3)
        want = P.forward(t, cfg, W)
        check(run(cfg, W, dtype, context_len=1500).feed(t, [1380, 1]), want, dtype)


@both
@pytest.mark.parametrize("heads", [20, 41, 75])
def test_heads_that_share_a_cluster(run, heads, dtype):  # noqa: F811
    cfg, W = B.latent_case(seed=heads, layers=1, mlp_none=(0,), mixer=dict(heads=heads, dim=10, rot_dim=4, vdim=9, kv_rank=37))
    t = B.tokens(cfg, 40, 3)
    check(run(cfg, W, dtype).feed(t, [1]), P.forward(t, cfg, W), dtype)
