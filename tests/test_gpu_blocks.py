"""Block models on the GPU against the plain implementation (tests/plain_blocks.py): each mechanism alone, whole stacks of
other sizes, prompts against token-by-token decoding, portions, reuse of a context, window and block edges, long decoding,
greedy generation, the replay program."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import block_cases as B
import plain_blocks as P
from block_runs import DTYPES, LIMIT, WHOLE, both, check, row_errors, run  # noqa: F401 (run: fixture)

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

# one mechanism at a time (a branch whose scale is zero adds nothing), and stacks of unequal sizes
CASES = {
    "attention": dict(layers=("parallel",), streams=1, mixer=dict(right_scale=0.0), mlp_none=(0,)),
    "attention, one kv head": dict(layers=("parallel",), mixer=dict(right_scale=0.0, heads=3, kv_heads=1, dim=17, vdim=33), mlp_none=(0,)),
    "attention, no groups": dict(layers=("parallel",), mixer=dict(right_scale=0.0, heads=2, kv_heads=2, dim=64, vdim=128), mlp_none=(0,)),
    "attention, wide heads": dict(layers=("parallel",), mixer=dict(right_scale=0.0, heads=2, kv_heads=1, dim=144, vdim=40), mlp_none=(0,)),
    "attention, blocks of one": dict(layers=("parallel",), mixer=dict(right_scale=0.0, window=6, pool=1), mlp_none=(0,)),
    "attention, window of one": dict(layers=("parallel",), mixer=dict(right_scale=0.0, window=1, pool=3), mlp_none=(0,)),
    "attention, blocks longer than the window": dict(layers=("parallel",), mixer=dict(right_scale=0.0, window=5, pool=19), mlp_none=(0,)),
    "retention": dict(layers=("parallel",), streams=1, mixer=dict(left_scale=0.0), mlp_none=(0,)),
    "retention, all dimensions turn": dict(layers=("parallel",), mixer=dict(left_scale=0.0, rheads=1, rdim=40, rvdim=72, rot_dims=40, base=10000.0), mlp_none=(0,)),
    "retention, two dimensions turn": dict(layers=("parallel",), mixer=dict(left_scale=0.0, rheads=5, rdim=70, rvdim=7, rot_dims=2, decay=[0.5, 0.9, 0.99, 1.0, 0.97]), mlp_none=(0,)),
    "retention, large state": dict(layers=("parallel",), mixer=dict(left_scale=0.0, rheads=2, rdim=160, rvdim=136, rot_dims=64), mlp_none=(0,)),
    "wkv": dict(layers=("wkv",), streams=1, mlp_none=(0,)),
    "wkv, one head": dict(layers=("wkv",), wkv=dict(heads=1, dim=130), mlp_none=(0,)),
    "wkv, many heads": dict(layers=("wkv",), wkv=dict(heads=9, dim=32), mlp_none=(0,)),
    "feed-forward after wkv": dict(layers=("wkv",), streams=1, ff=40),
    "two streams": dict(layers=("parallel", "wkv"), streams=2),
    "four streams": dict(layers=("wkv", "parallel"), streams=4, width=100),
    "eight streams": dict(layers=("parallel", "wkv"), streams=8, width=70),
    "loop": dict(layers=("wkv", "parallel", "wkv"), loop={"start": 0, "stop": 2, "times": 3}, mlp_none=(1,)),
    "loop over the end": dict(layers=("parallel", "wkv"), loop={"start": 1, "stop": 2, "times": 2}, vocab=1003, buckets=7),
    "wider": dict(layers=("parallel", "wkv"), width=384, ff=640, mixer=dict(heads=6, kv_heads=3, dim=64, vdim=64, window=40, pool=8, rheads=4, rdim=64, rvdim=64, rot_dims=64), wkv=dict(heads=6, dim=64)),
}


@both
@pytest.mark.parametrize("name", sorted(CASES))
def test_against_plain_whole_and_token_by_token(run, name, dtype):
    # (seeds with which a first token's heads are far from zero: their normalisation would amplify bfloat16 rounding)
    cfg, W = B.case(seed=23 if name == "loop" else len(name), **CASES[name])
    t = B.tokens(cfg, 75, len(name))
    want = P.forward(t, cfg, W)
    r = run(cfg, W, dtype)
    check(r.feed(t, WHOLE), want, dtype)
    check(r.feed(t, [1]), want, dtype)  # every token through the captured step
    check(r.feed(t, [30, 1]), want, dtype)


@both
@pytest.mark.parametrize("cuts", [[2], [3, 2, 7], [16], [17, 1, 1, 2], [64, 2], [5, 1, 30]])
def test_portions(run, cuts, dtype):
    cfg, W = B.case(seed=9, layers=("parallel", "wkv", "parallel"), loop={"start": 0, "stop": 2, "times": 2})
    t = B.tokens(cfg, 90, 3)
    check(run(cfg, W, dtype).feed(t, cuts), P.forward(t, cfg, W), dtype)


@both
def test_context_is_reused_by_the_next_sequence(run, dtype):
    cfg, W = B.case(seed=4, layers=("parallel", "wkv"))
    r = run(cfg, W, dtype)
    for i, (n, cuts) in enumerate([(80, WHOLE), (1, [1]), (33, [2]), (70, [1]), (5, WHOLE), (2, [1])]):
        t = B.tokens(cfg, n, 20 + i)
        check(r.feed(t, cuts), P.forward(t, cfg, W), dtype)


@both
def test_first_tokens(run, dtype):
    cfg, W = B.case(seed=6, layers=("wkv", "parallel"))
    r = run(cfg, W, dtype)
    for n in (1, 2, 3, 4):
        t = B.tokens(cfg, n, n)
        want = P.forward(t, cfg, W)
        check(r.feed(t, WHOLE), want, dtype)
        check(r.feed(t, [1]), want, dtype)
    # the first token takes the bigram row of its own: another row gives other logits
    other = copy.deepcopy(W)
    other["bigram"][-1] = other["bigram"][0]
    t = B.tokens(cfg, 3, 1)
    assert row_errors(P.forward(t, cfg, other), P.forward(t, cfg, W))[0] > 5 * LIMIT["bfloat16"]


def standout_case(window, pool, seed=2):
    """One attention layer in which token 0's key dwarfs all others for every query: whoever sees it shows it."""
    cfg, W = B.case(seed=seed, layers=("parallel",), streams=1, mlp_none=(0,), buckets=1,
                    mixer=dict(right_scale=0.0, window=window, pool=pool, heads=2, kv_heads=1, dim=16, vdim=16, scale=0.25))
    W["bigram"][:] = 0
    w = cfg["width"]
    W["embed"][:, 0], W["embed"][:, 1] = 3.0, 0.0   # channel 0: the same in every token, channel 1: token 0 only
    W["embed"][0, 1] = 6.0
    W["l0.norm1"][:] = 0
    W["l0.mix.left.q"][:], W["l0.mix.left.k"][:] = 0, 0
    W["l0.mix.left.q"][::16, 0] = 4.0
    W["l0.mix.left.k"][0, 1] = 4.0
    W["l0.mix.left.o"] *= 4
    return cfg, W


@both
@pytest.mark.parametrize("window,pool", [(13, 4), (64, 16), (20, 7)])
def test_window_and_block_edges(run, window, pool, dtype):
    cfg, W = standout_case(window, pool)
    n = 5 * window + 3 * pool
    wrong = []
    for d in (-1, 1):  # a window one off, blocks one off
        c = copy.deepcopy(cfg)
        c["layers"][0]["mixer"]["left"]["mask"]["size"] += d
        wrong.append(c)
    c = copy.deepcopy(cfg)
    c["layers"][0]["mixer"]["left"]["mask"]["pool"] = 10 ** 6
    wrong.append(c)
    r = run(cfg, W, dtype, context_len=512)
    for at in (0, pool - 1, pool, 2 * pool + 1, window):
        t = [1 + x % (cfg["vocab"] - 1) for x in B.tokens(cfg, n, at)]
        t[at] = 0
        want = P.forward(t, cfg, W)
        for c in wrong:  # each of these mistakes is far outside the limit somewhere
            assert row_errors(P.forward(t, c, W), want).max() > 3 * LIMIT["bfloat16"]
        for cuts in (WHOLE, [1], [window, 1], [at + 1, 2]):
            check(r.feed(t, cuts), want, dtype)


@both
def test_far_key_through_a_block_mean_and_a_state(run, dtype):
    """A token hundreds of positions back is still seen (its block's mean, the recurrent states), and its loss would show."""
    cfg, W = standout_case(32, 4)
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
def test_long_decoding(run, dtype):
    cfg, W = B.case(seed=8, layers=("parallel", "wkv"), mixer=dict(window=24, pool=8))
    t = B.tokens(cfg, 420, 7)
    check(run(cfg, W, dtype, context_len=430).feed(t, [4, 1]), P.forward(t, cfg, W), dtype)


def test_passes_longer_than_the_row_buffers(run):
    cfg, W = B.case(seed=12, layers=("parallel", "wkv"), width=40, ff=24, vocab=64, streams=2,
                    mixer=dict(heads=1, kv_heads=1, dim=8, vdim=8, window=100, pool=16, rheads=1, rdim=8, rvdim=8, rot_dims=8), wkv=dict(heads=1, dim=8))
    t = B.tokens(cfg, 2500, 2)
    want = P.forward(t, cfg, W)
    for dtype in DTYPES:
        r = run(cfg, W, dtype, context_len=2600)
        check(r.feed(t, WHOLE), want, dtype, factor=2.0 if dtype == "bfloat16" else 1.0)  # (a narrow model averages little out)


@pytest.mark.parametrize("keys", [{"block_attn_mma": 0}, {"block_row_one_cta": 0}, {"prefill_gate_fused": 256}, {"prefill_gate_fused": 512}, {"prefill_tc_sk": 256},
                                  {"prefill_tc_pair": 128}, {"use_graph": 0, "use_pdl": 0}])
def test_kernel_choices_agree(lcu, run, keys):
    """Other kernels for the same products and attention: balanced and two-SM products, the gate in the product's epilogue,
    the per-row attention, steps without a graph."""
    defaults = {"block_attn_mma": 1, "block_row_one_cta": 2048, "prefill_gate_fused": -1, "prefill_tc_sk": -1, "prefill_tc_pair": -1, "use_graph": 1, "use_pdl": 1}
    cfg, W = B.case(seed=14, layers=("parallel", "wkv"), width=256, ff=512,
                    mixer=dict(heads=4, kv_heads=2, dim=64, vdim=64, window=48, pool=16, rheads=2, rdim=64, rvdim=64, rot_dims=64), wkv=dict(heads=4, dim=64))
    t = B.tokens(cfg, 300, 4)
    want = P.forward(t, cfg, W)
    try:
        for k, v in keys.items():
            lcu.check(lcu.lib.lcu_set_tuning(k.encode(), v))
        check(run(cfg, W, "bfloat16", context_len=512).feed(t, [290, 1]), want, "bfloat16")
    finally:
        for k in keys:
            lcu.check(lcu.lib.lcu_set_tuning(k.encode(), defaults[k]))


def test_single_stream_without_tensors_is_the_plain_residual(run):
    cfg, W = B.case(seed=15, layers=("parallel", "wkv"), streams=1)
    for k in [k for k in W if ".hc" in k]:
        W[k] = np.ones_like(W[k])
    bare = {k: v for k, v in W.items() if ".hc" not in k}
    t = B.tokens(cfg, 40, 1)
    check(run(cfg, bare, "float32").feed(t, WHOLE), P.forward(t, cfg, W), "float32")


def test_greedy_generation(lcu, run):
    """next_token and the device-chained loop pick the plain implementation's argmax, token after token."""
    cfg, W = B.case(seed=16, layers=("parallel", "wkv"), loop={"start": 0, "stop": 2, "times": 2})
    r = run(cfg, W, "float32")
    prompt = B.tokens(cfg, 12, 9)
    seq = list(prompt)
    for _ in range(16):
        seq.append(int(P.forward(seq, cfg, W)[-1].argmax()))
    want = seq[len(prompt):]
    r.ctx.clear_tokens()
    got = [r.ctx.next_token(prompt)]
    while len(got) < 16:
        got.append(r.ctx.next_token([got[-1]]))
    assert got == want
    r.ctx.clear_tokens()
    first = r.ctx.next_token(prompt)
    toks, ms = r.ctx.decode_chained(first, 15)
    assert [first] + toks.tolist() == want and ms > 0
    p = r.ctx.probs().view(np.float16).astype(np.float64)
    lg = P.forward(seq[:-1], cfg, W)[-1]
    e = np.exp(lg - lg.max())
    assert np.abs(p - e / e.sum()).max() < 2e-3
    assert r.ctx.tokens_left() == 256 - len(prompt) - 15


def test_sampling_repeats_for_a_seed(run):
    cfg, W = B.case(seed=17)
    r = run(cfg, W, "bfloat16")
    W["head"] *= 0.2
    seen = []
    for seed in (5, 5, 6):
        r.ctx.clear_tokens()
        r.ctx.set_sampling(1, seed)
        t = r.ctx.next_token(B.tokens(cfg, 6, 3))
        seen.append([t] + r.ctx.decode_chained(t, 20)[0].tolist())
    assert seen[0] == seen[1] != seen[2]


def test_errors(lcu, run, tmp_path):
    cfg, W = B.case(seed=18)
    r = run(cfg, W, "bfloat16", context_len=16)
    with pytest.raises(lcu.LcuError, match="context length"):
        r.ctx.step(B.tokens(cfg, 17))
    with pytest.raises(lcu.LcuError, match="vocabulary"):
        r.ctx.step([cfg["vocab"]])
    with pytest.raises(lcu.LcuError, match="outside"):
        r.ctx.step([1, 2], [2])
    with pytest.raises(lcu.LcuError, match="LLaMA"):
        r.model.save(str(tmp_path))
    r.ctx.step([1, 2, 3])
    with pytest.raises(lcu.LcuError, match="recurrent"):
        r.ctx.rollover(1)
    gone = dict(W)
    gone.pop("l0.norm2")
    with pytest.raises(lcu.LcuError, match="l0.norm2"):
        lcu.Model.load(B.write(tmp_path / "a", cfg, gone))
    gone = dict(W, head=W["head"][:-1])
    with pytest.raises(lcu.LcuError, match="head"):
        lcu.Model.load(B.write(tmp_path / "b", cfg, gone))
    assert r.model.family() == "Filulix"


def test_llama_step_gives_the_last_logits(lcu):
    m = lcu.Model.synthetic(dim=256, n_heads=2, n_layers=2, n_vocab=1000, seed=3, scale=0.08)
    c = lcu.Context(m, context_len=32)
    lg, tok = c.step([5, 6, 7], [2], token=True)
    assert tok == int(lg[0].argmax()) and m.family() == "llama"
    lg, tok = c.step([tok], [0], token=True)
    assert tok == int(lg[0].argmax())
    with pytest.raises(lcu.LcuError, match="last token"):
        c.step([5, 6, 7], [0])
    c.close()
    m.close()


@both
def test_replay_program(tmp_path, dtype):
    cfg, W = B.case(seed=19, layers=("parallel", "wkv"))
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
            check(np.fromfile(f, np.float32).reshape(len(w), cfg["vocab"]), w, dtype)
