"""Small Boketar configurations for the tests.  Between them every size differs, and sizes that are often equal are not
(key and value size, heads of the two sides of a pair, query/key heads and value heads of the delta rule, the two narrow
inner widths, the taps of the two kinds of convolution); every layer type comes with and without a feed-forward."""


def window(heads, kv_heads, dim, vdim, conv, size, scale, base, dims):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale,
            "mask": {"size": size}, "rot": {"base": base, "dims": dims}}


def lightning(heads, dim, vdim, decay):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}


def pair(left, right, ff):
    return {"type": "parallel", "mixer": {"left": left, "right": right},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def delta(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank, ff=None):
    return {"type": "channel_delta",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv,
                      "decay_rank": decay_rank, "gate_rank": gate_rank},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def model(vocab, width, streams, eps, scale, layers):
    return {"architecture": "Boketar", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
            "embedding": {"scale": scale}, "layers": layers}


# three streams; a pair first (6 query heads on 3, key 24 against value 40, a window of 21 that is no multiple of a page,
# 8 of 24 coordinates rotated), a delta rule with three value heads on one query/key head and a feed-forward
BOKETAR_A = model(211, 64, 3, 1e-5, 3.0, [
    pair(window(6, 3, 24, 40, 3, 21, 0.2, 5000.0, 8), lightning(3, 16, 8, [0.9, 0.97, 0.995]), 72),
    delta(3, 1, 16, 24, 4, 6, 10, ff=40),
    pair(window(2, 1, 32, 16, 2, 50, 0.18, 90000.0, 32), lightning(5, 8, 12, [0.5, 0.8, 0.99, 0.999, 1.0]), None),
    delta(2, 2, 32, 8, 2, 3, 1),
])
# two streams; convolutions of ONE tap (no inputs kept) in either kind of layer, a window of one (a row sees itself), two
# rotated coordinates, one lightning head, a delta rule with long keys and five taps
BOKETAR_B = model(320, 96, 2, 1e-6, 0.5, [
    delta(4, 2, 40, 16, 1, 16, 8),
    pair(window(4, 1, 16, 24, 1, 1, 0.4, 100.0, 2), lightning(1, 64, 32, [0.99]), 56),
    delta(2, 1, 136, 40, 5, 9, 7, ff=24),
    pair(window(3, 3, 80, 8, 4, 33, 0.11, 1000.0, 80), lightning(2, 40, 24, [0.95, 0.9995]), None),
])
# a width that is no multiple of 8 (no tensor-core product), five streams, an odd vocabulary, head sizes that are no
# multiple of 4, more taps than a portion has rows, a window wider than any test sequence
BOKETAR_C = model(97, 42, 5, 3e-6, 2.0, [
    pair(window(3, 1, 20, 12, 7, 400, 0.25, 777.0, 6), lightning(1, 12, 20, [0.9]), 20),
    delta(2, 1, 6, 10, 3, 2, 5, ff=12),
    delta(1, 1, 3, 5, 8, 1, 2),
])
# one stream (the residual's weights still apply)
BOKETAR_D = model(64, 32, 1, 1e-5, 1.0, [
    delta(2, 2, 8, 8, 2, 4, 4, ff=16),
    pair(window(2, 2, 8, 16, 2, 12, 0.35, 50.0, 4), lightning(2, 8, 16, [0.7, 0.98]), 24),
])
CONFIGS = {"A": BOKETAR_A, "B": BOKETAR_B, "C": BOKETAR_C, "D": BOKETAR_D}
