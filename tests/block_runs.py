"""What the GPU tests of the block models share: a loaded model with a context, limits, comparison of logits."""
import numpy as np
import pytest

import block_cases as B

LIMIT = {"float32": 1e-5, "bfloat16": 4e-2}  # RMS error of a row of logits, as a share of the RMS of all expected logits


def row_errors(got, want):
    d = np.asarray(got, np.float64) - want
    return np.sqrt((d * d).mean(1)) / np.sqrt((want * want).mean())


def check(got, want, dtype, factor=1.0):
    e = row_errors(got, want)
    assert np.isfinite(e).all() and e.max() <= LIMIT[dtype] * factor, (float(e.max()), int(e.argmax()))


class Running:
    """A model directory loaded in one number format, with one context."""

    def __init__(self, lcu, path, dtype, context_len=256):
        self.model = lcu.Model.load(path, dtype=dtype)
        self.ctx = lcu.Context(self.model, context_len=context_len, temperature=1.0)

    def feed(self, toks, cuts):
        """All logits of a sequence fed in portions of the given sizes (the last size repeats)."""
        self.ctx.clear_tokens()
        out, at, i = [], 0, 0
        while at < len(toks):
            n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
            out.append(self.ctx.step(toks[at:at + n], list(range(n))))
            at, i = at + n, i + 1
        return np.concatenate(out)

    def close(self):
        self.ctx.close()
        self.model.close()


@pytest.fixture
def run(lcu, tmp_path):
    made = []

    def make(cfg, W, dtype, context_len=256):
        made.append(Running(lcu, B.write(tmp_path / f"m{len(made)}", cfg, W), dtype, context_len))
        return made[-1]

    yield make
    for r in made:
        r.close()


WHOLE = [1 << 20]
DTYPES = ["float32", "bfloat16"]
both = pytest.mark.parametrize("dtype", DTYPES)
