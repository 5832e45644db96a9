"""Merusun configurations drawn from a seed: one to six layers of any kind in any order, readers of earlier keys with
windows of their own, 1 to 12 heads, head sizes that are and are not multiples of 4, latents of 6 to 200 with rotated parts
of 2 to 64, windows of 1 to 300, caps of 0.5 to 40, up to 16 experts in groups, pages of 4 to 64.  Every configuration runs
whole, in portions and token by token, in 32-bit and in bfloat16, against the plain implementation."""
import random

import pytest
import torch

import helpers
import merusun_configs as mc
import plain_merusun as plain
from test_gezozen_engine_gpu import Tally, check, make_runner
from test_merusun_engine_gpu import TOL32, tolerance, write_folder

pytestmark = pytest.mark.gpu


def draw(seed):
    r = random.Random(seed)

    def mlp():
        if r.random() < 0.3:
            return None
        count = r.choice([1, 1, 2, 3, 4])
        each, keep = r.randint(1, 16 // count), r.randint(1, count)
        return mc.moe(r.choice([8, 12, 32, 56, 96]), count * each, r.randint(1, min(each * keep, 8)), count, keep,
                      r.choice([1.0, 0.5, 2.5]), r.choice([None, 8, 20, 64]))
    layers = []
    for i in range(r.randint(1, 6)):
        kind = r.random()
        own = [j for j, L in enumerate(layers) if L["type"] == "attention" and "kv_from" not in L["mixer"]]
        window = r.choice([1, 2, 7, 16, 40, 300])
        if kind < 0.35:
            layers.append(mc.memory(r.randint(1, 6), r.choice([2, 5, 12, 16, 32, 72, 128, 160]), r.choice([1, 3, 6, 8, 32, 72]),
                                    r.choice([0.5, 3.0, 15.0, 40.0]), mlp()))
        elif kind < 0.65:
            dim, rot = r.choice([6, 8, 20, 32, 64, 128]), r.choice([2, 6, 8, 16, 64])
            layers.append(mc.latent(r.choice([1, 2, 3, 5, 8, 12]), dim, rot, r.choice([4, 10, 16, 64, 128]),
                                    r.choice([6, 16, 40, 64, 120, 200]), window, (dim + rot) ** -0.5, r.choice([50.0, 1e4, 1e6]), mlp()))
        elif own and kind < 0.85:
            j = r.choice(own)
            m = layers[j]["mixer"]
            layers.append(mc.attention(m["heads"], m["kv_heads"], m["dim"], m["vdim"], window, r.choice([0.1, 0.3]), j, mlp()))
        else:
            g = r.choice([1, 2, 3])
            layers.append(mc.attention(g * r.choice([1, 2, 4]), g, r.choice([8, 12, 20, 32, 64, 96, 128, 144]),
                                       r.choice([6, 8, 40, 64, 80, 128]), window, r.choice([0.1, 0.3]), None, mlp()))
    return mc.model(r.choice([53, 128, 300]), r.choice([24, 40, 64, 96, 128, 50]), r.choice([1e-5, 1e-6, 1e-2]),
                    r.choice([0.5, 2.0, 8.0]), layers)


@pytest.mark.parametrize("seed", range(12))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_drawn_configuration(tmp_path, seed, dtype):
    from allpaca_b200.engine.batch import BatchEntry
    config = draw(3000 + seed) if dtype == "float32" else mc.every_expert(draw(3000 + seed))
    weights = write_folder(tmp_path, config, seed=seed, dtype=dtype)
    r = random.Random(seed)
    seqs = {k: helpers.random_tokens(n, config["vocab"], 10 * seed + k) for k, n in enumerate([r.randint(40, 90), 1, 19])}
    want = {k: plain.forward(weights, config, t) for k, t in seqs.items()}
    runner = make_runner(tmp_path, dtype, 256, page_size=r.choice([4, 8, 16, 64]), max_seqs=3)
    tally, tol = Tally(), tolerance(dtype, weights, config, [seqs[0]])
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
