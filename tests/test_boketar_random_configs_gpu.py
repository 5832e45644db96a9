"""Boketar configurations drawn from a seed: one to six layers of either kind in any order, with and without a
feed-forward, 1 to 8 streams, 1 to 12 heads, head sizes that are and are not multiples of 4, rotations of 2 coordinates up
to the whole head, windows of 1 to 300, convolutions of 1 to 9 taps, narrow pairs of 1 to 33, pages of 4 to 64.  Every
configuration runs whole, in portions and token by token, in 32-bit and in bfloat16, against the plain implementation.

How far bfloat16's rounding moves the logits differs from draw to draw by a factor of ten (small widths, many layers, an
embedding that weighs little beside them), so each draw has its own tolerance: twice the largest row error that the
plain implementation shows when it rounds what the engine stores."""
import random

import pytest
import torch

import boketar_configs as bc
import helpers
import plain_boketar as plain
from test_boketar_engine_gpu import TOL, write_folder
from test_gezozen_engine_gpu import Tally, check, make_runner

pytestmark = pytest.mark.gpu


def draw(seed):
    r = random.Random(seed)

    def ff():
        return r.choice([None, 8, 20, 48, 96])

    def layer():
        g = r.choice([1, 2, 3])
        if r.random() < 0.5:
            return bc.delta(g * r.choice([1, 2, 4]), g, r.choice([2, 5, 12, 16, 32, 72, 128, 160]), r.choice([3, 6, 8, 32, 72]),
                            r.randint(1, 6), r.choice([1, 3, 8, 33]), r.choice([1, 5, 16, 24]), ff())
        dim = r.choice([8, 12, 20, 32, 64, 96, 128, 144])
        left = bc.window(g * r.choice([1, 2, 4]), g, dim, r.choice([6, 8, 40, 64, 80, 128]), r.choice([1, 2, 3, 5, 9]),
                         r.choice([1, 2, 7, 16, 40, 300]), r.choice([0.1, 0.25, dim ** -0.5]), r.choice([50.0, 10000.0]),
                         r.choice([2, dim, max(2, dim // 4 * 2)]))
        heads = r.randint(1, 6)
        right = bc.lightning(heads, r.choice([3, 6, 8, 16, 48, 64]), r.choice([4, 10, 32, 64]),
                             [1.0 - 2.0 ** -r.randint(1, 11) for _ in range(heads)])
        return bc.pair(left, right, ff())
    return bc.model(r.choice([53, 128, 300]), r.choice([24, 40, 64, 96, 128, 50]), r.choice([1, 2, 3, 4, 5, 8]),
                    r.choice([1e-5, 1e-6, 3e-6]), r.choice([0.5, 1.0, 2.0]), [layer() for _ in range(r.randint(1, 6))])


@pytest.mark.parametrize("seed", range(10))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_drawn_configuration(tmp_path, seed, dtype):
    from allpaca_b200.engine.batch import BatchEntry
    config = draw(2000 + seed)
    weights = write_folder(tmp_path, config, seed=seed, dtype=dtype)
    r = random.Random(seed)
    seqs = {k: helpers.random_tokens(n, config["vocab"], 10 * seed + k) for k, n in enumerate([r.randint(40, 90), 1, 19])}
    want = {k: plain.forward(weights, config, t) for k, t in seqs.items()}
    runner = make_runner(tmp_path, dtype, 256, page_size=r.choice([4, 8, 16, 64]), max_seqs=3)
    tally, tol = Tally(), TOL[dtype]
    if dtype == "bfloat16":
        with plain.rounded(torch.bfloat16):
            off = plain.forward(weights, config, seqs[0]) - want[0]
        tol = 2.0 * float((off ** 2).mean(-1).sqrt().max() / (want[0] ** 2).mean().sqrt())
    # whole; then two requests side by side in portions of any size and single rows
    for k, toks in seqs.items():
        check(runner.step([BatchEntry(("w", k), toks, list(range(len(toks))))]), want[k], tol, (seed, "whole", k), tally)
        runner.finish(("w", k))
    at = {0: 0, 2: 0}
    while any(at[k] < len(seqs[k]) for k in at):
        entries, rows = [], []
        for k in at:
            if at[k] < len(seqs[k]):
                n = min(r.choice([1, 1, 2, 5, 17]), len(seqs[k]) - at[k])
                entries.append(BatchEntry(k, seqs[k][at[k]:at[k] + n], list(range(n))))
                rows.append((k, at[k], n))
                at[k] += n
        logits = runner.step(entries)
        row = 0
        for k, a, n in rows:
            check(logits[row:row + n], want[k][a:a + n], tol, (seed, "portion", k, a, n), tally)
            row += n
    tally.finish((seed, dtype))
    runner.finish(0)
    runner.finish(2)
    runner.cache.check()
