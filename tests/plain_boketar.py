"""The Boketar decoder restated plainly: one function per mechanism, float64, token by token where the design is a
recurrence.  Nothing here is shared with the engine; tests compare the engine against it.

A model is ``(cfg, W)``: ``cfg`` the dictionary of config.json and ``W`` a dictionary of float64 tensors by
checkpoint name.  Every function takes whole sequences ``[T, ...]`` of ONE request, positions ``0 .. T-1``.
"""
from __future__ import annotations

import contextlib
import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64
UNIT_EPS = 1e-6                # under the root where the delta rule makes queries and keys unit vectors


_ROUND: List[Optional[torch.dtype]] = [None]


@contextlib.contextmanager
def rounded(dtype):
    """Within: what an engine of that storage type rounds is rounded (the inputs of products, queries, keys and values), all
    else stays exact.  How far this moves the logits of a model says how closely such an engine can follow it."""
    _ROUND[0] = dtype
    try:
        yield
    finally:
        _ROUND[0] = None


def stored(x):
    return x if _ROUND[0] is None else x.to(_ROUND[0]).to(F64)


def lin(W, name, x, bias=False):
    y = stored(x) @ W[name].T
    return y + W[name + ".b"] if bias else y


def silu(z):
    return z * torch.sigmoid(z)


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    """The layers' norm: the weight is stored around zero and counts as ``1 + w``."""
    return rms(x, eps) * (1.0 + w)


# ---- hyper-connections ------------------------------------------------------------------------
def widen(x, streams):
    """``[T, W]`` -> ``[T, streams, W]``, all streams alike."""
    return x[:, None, :].repeat(1, streams, 1)


def gather_streams(xs, w_in):
    """What a sublayer's norm reads: the streams weighted by one number each."""
    return torch.einsum("tsw,s->tw", xs, w_in)


def scatter_streams(xs, y, w_out, w_mix):
    """All streams at once from the old ones: ``new[t] = sum_s mix[s, t] old[s] + out[t] y`` (``mix`` [from, to])."""
    return torch.einsum("tsw,so->tow", xs, w_mix) + y[:, None, :] * w_out[None, :, None]


# ---- short convolution, rotation, attention ---------------------------------------------------
def short_conv(x, w):
    """``x [T, C]``, ``w [C, taps]``: every channel filtered along time, the last tap on the row itself, zeros before
    the start."""
    T, C = x.shape
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=F64), x], dim=0)
    y = torch.zeros(T, C, dtype=F64)
    for j in range(taps):
        y = y + padded[j:j + T] * w[:, j]
    return y


def rotate(x, rot, positions):
    """``x [T, heads, dim]``: pairs of NEIGHBOURING coordinates (2i, 2i+1) among the first ``dims`` turned by
    ``p * base^(-2i/dims)``; the rest of the head passes."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    ang = positions.to(F64)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def attend(q, k, v, scale, window, sink):
    """``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, V]``: row i over the keys ``i - window + 1 .. i`` (None: all up to
    i); the softmax's denominator also holds ``exp(sink[h])``, to which no value belongs (None: no sink)."""
    q, k, v = stored(q), stored(k), stored(v)
    T, H, _ = q.shape
    G = k.shape[1]
    pos = torch.arange(T)
    dist = pos[:, None] - pos[None, :]
    seen = dist >= 0
    if window is not None:
        seen = seen & (dist < window)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for a in range(H):
        g = a // (H // G)
        s = ((q[:, a] @ k[:, g].T) * scale).masked_fill(~seen, -math.inf)
        if sink is not None:
            s = torch.cat([s, sink[a].expand(T, 1)], dim=1)
        p = torch.softmax(s, dim=-1)[:, :T]
        out[:, a] = p @ v[:, g]
    return out


def window_attention(W, p, m, h):
    """The left side of a pair: biased projections, short convolutions (no activation), rotation, window, sink."""
    T = h.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(T)
    q = short_conv(lin(W, p + "q", h, True), W[p + "q.conv"]).reshape(T, H, D)
    k = short_conv(lin(W, p + "k", h, True), W[p + "k.conv"]).reshape(T, G, D)
    v = short_conv(lin(W, p + "v", h, True), W[p + "v.conv"]).reshape(T, G, V)
    q, k = rotate(q, m["rot"], pos), rotate(k, m["rot"], pos)
    out = attend(q, k, v, float(m["scale"]), int(m["mask"]["size"]), W[p + "sink"])
    return lin(W, p + "o", out.reshape(T, H * V), True)


# ---- recurrences ------------------------------------------------------------------------------
def lightning_attention(W, p, m, h, eps):
    """The right side of a pair: SiLU on queries, keys and values, one fixed decay per head; the heads' read-outs
    normed TOGETHER, under a sigmoid gate."""
    T = h.shape[0]
    H, D, V = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = silu(lin(W, p + "q", h)).reshape(T, H, D)
    k = silu(lin(W, p + "k", h)).reshape(T, H, D)
    v = silu(lin(W, p + "v", h)).reshape(T, H, V)
    decay = torch.tensor([float(d) for d in m["decay"]], dtype=F64)
    S = torch.zeros(H, D, V, dtype=F64)
    o = torch.zeros(T, H, V, dtype=F64)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    o = rms(o.reshape(T, H * V), eps) * W[p + "norm"]
    return lin(W, p + "o", o * torch.sigmoid(lin(W, p + "g", h)))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def channel_decay(W, p, m, h):
    """One decay per head and key channel: ``exp(-exp(A_log[head]) softplus(W_a2 W_a1 h + dt_bias))``, [T, H, D]."""
    H, D = int(m["heads"]), int(m["dim"])
    z = lin(W, p + "a2", lin(W, p + "a1", h)) + W[p + "dt_bias"]
    z = torch.nn.functional.softplus(z).reshape(-1, H, D)
    return torch.exp(-torch.exp(W[p + "A_log"])[None, :, None] * z)


def delta_recurrence(q, k, v, decay, beta):
    """``q, k [T, G, D]``, ``v [T, H, V]``, ``decay [T, H, D]``, ``beta [T, H]``: the state's rows forget channel by
    channel, then the state is corrected towards the value along the key; the read-out sees the correction."""
    T, H, V = v.shape
    rep = H // q.shape[1]
    S = torch.zeros(H, q.shape[2], V, dtype=F64)
    o = torch.zeros(T, H, V, dtype=F64)
    for t in range(T):
        kt, qt = k[t].repeat_interleave(rep, dim=0), q[t].repeat_interleave(rep, dim=0)
        S = decay[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, kt))
        S = S + kt[:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, qt)
    return o


def channel_delta(W, p, m, h, eps):
    """The delta rule with a decay per key channel and a sigmoid gate formed by a narrow pair of products."""
    T = h.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = silu(short_conv(lin(W, p + "q", h), W[p + "q.conv"])).reshape(T, G, D)
    k = silu(short_conv(lin(W, p + "k", h), W[p + "k.conv"])).reshape(T, G, D)
    v = silu(short_conv(lin(W, p + "v", h), W[p + "v.conv"])).reshape(T, H, V)
    o = delta_recurrence(unit(q) * D ** -0.5, unit(k), v, channel_decay(W, p, m, h), torch.sigmoid(lin(W, p + "b", h)))
    gate = torch.sigmoid(lin(W, p + "g2", lin(W, p + "g1", h)))
    o = (rms(o, eps) * W[p + "norm"]).reshape(T, H * V) * gate
    return lin(W, p + "o", o)


# ---- the layer --------------------------------------------------------------------------------
def normed_halves(a, b, wa, wb, eps):
    """Half the sum of two rows, each over its own root mean square and under its own plain weight."""
    return 0.5 * (rms(a, eps) * wa + rms(b, eps) * wb)


def mixer(W, cfg, i, h):
    L = cfg["layers"][i]
    eps = float(cfg["norm"]["eps"])
    p, m = f"l{i}.mix.", L["mixer"]
    if L["type"] == "channel_delta":
        return channel_delta(W, p, m, h, eps)
    left = window_attention(W, p + "left.", m["left"], h)
    right = lightning_attention(W, p + "right.", m["right"], h, eps)
    return normed_halves(left, right, W[p + "left.out"], W[p + "right.out"], eps)


def dense(W, p, h):
    return lin(W, p + "down", silu(lin(W, p + "gate", h)) * lin(W, p + "up", h))


def layer(W, cfg, i, xs):
    """``xs [T, streams, width]`` -> the same, after the layer's one or two sublayers."""
    eps = float(cfg["norm"]["eps"])
    p = f"l{i}."
    u = gather_streams(xs, W[p + "hc1.in"])
    y = mixer(W, cfg, i, norm(u, W[p + "norm1"], eps))
    xs = scatter_streams(xs, y, W[p + "hc1.out"], W[p + "hc1.mix"])
    if cfg["layers"][i].get("mlp") is not None:
        u = gather_streams(xs, W[p + "hc2.in"])
        y = dense(W, p + "mlp.", norm(u, W[p + "norm2"], eps))
        xs = scatter_streams(xs, y, W[p + "hc2.out"], W[p + "hc2.mix"])
    return xs


def forward(W, cfg, tokens, streams: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one request; ``streams`` (optional) collects all streams after every layer."""
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * float(cfg["embedding"]["scale"])
    xs = widen(x, int(cfg["streams"]))
    for i in range(len(cfg["layers"])):
        xs = layer(W, cfg, i, xs)
        if streams is not None:
            streams.append(xs)
    return lin(W, "head", norm(xs.sum(1), W["final.norm"], float(cfg["norm"]["eps"])))


def greedy(W, cfg, prompt, count: int) -> List[int]:
    toks = list(prompt)
    for _ in range(count):
        toks.append(int(forward(W, cfg, toks)[-1].argmax()))
    return toks[len(prompt):]


# ---- tensors ----------------------------------------------------------------------------------
def tensor_shapes(cfg) -> Dict[str, tuple]:
    """Every tensor a model folder of this design holds, with its shape.  The inner widths of the two narrow pairs
    are in the mixer's ``decay_rank`` and ``gate_rank`` (a folder of another origin has them in the tensors alone)."""
    Wd, vocab, s = int(cfg["width"]), int(cfg["vocab"]), int(cfg["streams"])
    out = {"embed": (vocab, Wd), "final.norm": (Wd,), "head": (vocab, Wd)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        out[p + "norm1"] = (Wd,)
        out.update({p + "hc1.in": (s,), p + "hc1.out": (s,), p + "hc1.mix": (s, s)})
        if L["type"] == "channel_delta":
            H, G, D, V, taps = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
            ra, rg = int(m["decay_rank"]), int(m["gate_rank"])
            q = p + "mix."
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * V)):
                out.update({q + n: (rows, Wd), q + n + ".conv": (rows, taps)})
            out.update({q + "b": (H, Wd), q + "A_log": (H,), q + "norm": (V,), q + "a1": (ra, Wd), q + "a2": (H * D, ra),
                        q + "dt_bias": (H * D,), q + "g1": (rg, Wd), q + "g2": (H * V, rg), q + "o": (Wd, H * V)})
        else:
            l, r = m["left"], m["right"]
            H, G, D, V, taps = (int(l[k]) for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
            q = p + "mix.left."
            for n, rows in (("q", H * D), ("k", G * D), ("v", G * V)):
                out.update({q + n: (rows, Wd), q + n + ".b": (rows,), q + n + ".conv": (rows, taps)})
            out.update({q + "sink": (H,), q + "o": (Wd, H * V), q + "o.b": (Wd,), q + "out": (Wd,)})
            H, D, V = (int(r[k]) for k in ("heads", "dim", "vdim"))
            q = p + "mix.right."
            out.update({q + "q": (H * D, Wd), q + "k": (H * D, Wd), q + "v": (H * V, Wd), q + "g": (H * V, Wd),
                        q + "o": (Wd, H * V), q + "norm": (H * V,), q + "out": (Wd,)})
        if L.get("mlp") is not None:
            F = int(L["mlp"]["ff"])
            out[p + "norm2"] = (Wd,)
            out.update({p + "hc2.in": (s,), p + "hc2.out": (s,), p + "hc2.mix": (s, s)})
            out.update({p + "mlp.gate": (F, Wd), p + "mlp.up": (F, Wd), p + "mlp.down": (Wd, F)})
    return out


def random_tensors(cfg, seed: int) -> Dict[str, torch.Tensor]:
    """Weights with which every mechanism shows in the logits: matrices of unit gain, norm weights around what they
    stand for (zero for the layers' norms, one for the plain ones), streams that differ and mix, decays that neither
    die at once nor stay at 1, sinks of the size of the scores.  Rounded to bfloat16, so that a 16-bit checkpoint of
    them is exact."""
    g = torch.Generator().manual_seed(seed)
    s = int(cfg["streams"])
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        tail = name.rsplit(".", 1)[-1]
        if tail in ("norm1", "norm2") or name == "final.norm":
            t = 0.2 * torch.randn(shape, generator=g)
        elif tail in ("norm", "out") and ".hc" not in name:
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif tail == "in":
            t = (1.0 + 0.5 * torch.randn(shape, generator=g)) / s
        elif tail == "out":
            t = 1.0 + 0.5 * torch.randn(shape, generator=g)
        elif tail == "mix" and ".hc" in name:
            t = 0.6 * torch.eye(s) + 0.4 / s * (1.0 + torch.randn(shape, generator=g))
        elif name.endswith(".conv"):
            t = torch.randn(shape, generator=g) / shape[1] ** 0.5
        elif tail == "A_log":
            t = torch.log(0.05 + 0.5 * torch.rand(shape, generator=g))
        elif tail == "dt_bias":
            t = torch.randn(shape, generator=g) - 0.5
        elif tail == "sink":
            t = 1.0 + torch.randn(shape, generator=g)
        elif tail == "b" and len(shape) == 1:
            t = 0.3 * torch.randn(shape, generator=g)
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / shape[-1] ** 0.5
        out[name] = t.to(torch.bfloat16).to(F64)
    return out
