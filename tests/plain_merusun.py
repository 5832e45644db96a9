"""The Merusun decoder restated plainly: one function per mechanism, float64, token by token where the design is a
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
READ_EPS = 1e-6                # on the matrix memory's denominator


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


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


# ---- attention ----------------------------------------------------------------------------------
def visible(T, window):
    pos = torch.arange(T)
    dist = pos[:, None] - pos[None, :]
    seen = dist >= 0
    return seen if window is None else seen & (dist < window)


def attend(q, k, v, scale, window, one_in_denominator):
    """``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, V]``: row i over the keys ``i - window + 1 .. i`` (None: all up to
    i); with ``one_in_denominator`` the weights are ``exp(s_j) / (1 + sum exp(s))``, else an ordinary softmax."""
    q, k, v = stored(q), stored(k), stored(v)
    T, H, _ = q.shape
    G = k.shape[1]
    seen = visible(T, window)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for a in range(H):
        g = a // (H // G)
        s = ((q[:, a] @ k[:, g].T) * scale).masked_fill(~seen, -math.inf)
        top = s.max(dim=-1, keepdim=True).values
        if one_in_denominator:
            top = top.clamp(min=0.0)
        e = torch.exp(s - top)
        below = e.sum(-1, keepdim=True) + (torch.exp(-top) if one_in_denominator else 0.0)
        out[:, a] = (e / below) @ v[:, g]
    return out


def window_of(m):
    mask = m.get("mask")
    return int(mask["size"]) if mask else None


def keys_and_values(W, p, m, h, eps):
    """What a layer with projections of its own keeps: unit-mean-square keys and the values."""
    T = h.shape[0]
    G, D, V = int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    k = rms(lin(W, p + "k", h, True).reshape(T, G, D), eps)
    return k, lin(W, p + "v", h, True).reshape(T, G, V)


def attention(W, p, m, h, eps, kv):
    """Grouped-query attention without positions on ``kv`` (this layer's keys and values, or an earlier layer's)."""
    T = h.shape[0]
    H, D, V = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = rms(lin(W, p + "q", h, True).reshape(T, H, D), eps)
    out = attend(q, kv[0], kv[1], float(m["scale"]), window_of(m), True)
    return lin(W, p + "o", out.reshape(T, H * V))


def rotate(x, rot, positions):
    """``x [T, heads, dim]``: pairs of NEIGHBOURING coordinates (2i, 2i+1) among the first ``dims`` turned by
    ``p * base^(-2i/dims)``; the rest passes."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    ang = positions.to(F64)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def latent_attention(W, p, m, h, eps):
    """Per-head keys and values unfolded from one normed latent per token; a rotated key part that all heads share."""
    T = h.shape[0]
    H, D, E, V, R = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    pos = torch.arange(T)
    q = lin(W, p + "q", h).reshape(T, H, D + E)
    down = lin(W, p + "dkv", h)
    c = rms(down[:, :R], eps) * W[p + "dkv.norm"]
    turned = rotate(down[:, None, R:], m["rot"], pos)
    k = torch.cat([lin(W, p + "uk", c).reshape(T, H, D), turned.expand(T, H, E)], dim=-1)
    q = torch.cat([q[..., :D], rotate(q[..., D:], m["rot"], pos)], dim=-1)
    v = lin(W, p + "uv", c).reshape(T, H, V)
    out = attend(q, k, v, float(m["scale"]), window_of(m), False)
    return lin(W, p + "o", out.reshape(T, H * V))


# ---- matrix memory ------------------------------------------------------------------------------
def capped(z, cap):
    return cap * torch.tanh(z / cap)


def log_gates(W, p, m, h):
    """(log input gate, log forget gate), [T, H] each."""
    cap = float(m["gate_cap"])
    i = capped(lin(W, p + "i", h, True), cap)
    f = torch.nn.functional.logsigmoid(capped(lin(W, p + "f", h, True), cap))
    return i, f


def matrix_memory(q, k, v, i, f):
    """``q, k [T, H, D]``, ``v [T, H, V]``, log gates ``[T, H]``: a matrix and a vector per head, both scaled by
    ``exp(-m)`` of a running maximum ``m`` that starts at zero."""
    T, H, D = q.shape
    S, n, top = torch.zeros(H, D, v.shape[2], dtype=F64), torch.zeros(H, D, dtype=F64), torch.zeros(H, dtype=F64)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        new = torch.maximum(f[t] + top, i[t])
        keep, write = torch.exp(f[t] + top - new), torch.exp(i[t] - new)
        top = new
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        below = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-top)) + READ_EPS
        out[t] = torch.einsum("hdv,hd->hv", S, q[t]) / below[:, None]
    return out


def mlstm(W, p, m, h, eps):
    T = h.shape[0]
    H, D, V = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = lin(W, p + "q", h).reshape(T, H, D) * D ** -0.5
    k = lin(W, p + "k", h).reshape(T, H, D)
    v = lin(W, p + "v", h).reshape(T, H, V)
    o = rms(matrix_memory(q, k, v, *log_gates(W, p, m, h)), eps).reshape(T, H * V)
    return lin(W, p + "o", o * W[p + "norm"] * torch.sigmoid(lin(W, p + "g", h)))


# ---- feed-forward -------------------------------------------------------------------------------
def squared_relu(W, p, h):
    z = torch.relu(lin(W, p + ".up", h))
    return lin(W, p + ".down", z * z)


def route(z, r):
    """Router logits ``[T, experts]`` -> the chosen experts ``[T, top]`` and their weights.  Neighbouring experts form
    groups; a row chooses among the experts of its best groups (by a group's largest score) only."""
    s = torch.softmax(z, dim=-1)
    T, E = s.shape
    open_to = torch.ones(T, E, dtype=torch.bool)
    groups = r.get("groups")
    if groups:
        count, keep = int(groups["count"]), int(groups["keep"])
        best = s.reshape(T, count, E // count).max(-1).values.topk(keep, dim=-1).indices
        open_to = torch.zeros(T, count, dtype=torch.bool).scatter(1, best, True).repeat_interleave(E // count, dim=1)
    chosen = s.masked_fill(~open_to, -1.0).topk(int(r["top"]), dim=-1).indices
    return chosen, s.gather(1, chosen) * float(r["scale"])


def experts(W, p, mlp, h):
    chosen, weight = route(lin(W, p + "router", h), mlp["router"])
    out = torch.zeros_like(h)
    for e in range(int(mlp["router"]["experts"])):
        row, place = (chosen == e).nonzero(as_tuple=True)
        if len(row):
            out[row] += weight[row, place][:, None] * squared_relu(W, p + f"e{e}", h[row])
    if mlp.get("shared"):
        out = out + squared_relu(W, p + "shared", h)
    return out


# ---- the layer ----------------------------------------------------------------------------------
def layer(W, cfg, i, x, kept):
    """``kept``: the keys and values of the attention layers so far, by layer."""
    eps = float(cfg["norm"]["eps"])
    L, p = cfg["layers"][i], f"l{i}."
    m = L["mixer"]
    h = rms(x, eps) * W[p + "norm1"]
    if L["type"] == "mlstm":
        y = mlstm(W, p + "mix.", m, h, eps)
    elif L["type"] == "latent_attention":
        y = latent_attention(W, p + "mix.", m, h, eps)
    else:
        j = m.get("kv_from")
        if j is None:
            kept[i] = keys_and_values(W, p + "mix.", m, h, eps)
        y = attention(W, p + "mix.", m, h, eps, kept[i if j is None else j])
    x = x + rms(y, eps) * W[p + "norm1b"]
    if L.get("mlp") is not None:
        y = experts(W, p + "mlp.", L["mlp"], rms(x, eps) * W[p + "norm2"])
        x = x + rms(y, eps) * W[p + "norm2b"]
    return x


def forward(W, cfg, tokens, residual: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one request; ``residual`` (optional) collects the stream after every layer."""
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * float(cfg["embedding"]["scale"])
    kept: Dict[int, tuple] = {}
    for i in range(len(cfg["layers"])):
        x = layer(W, cfg, i, x, kept)
        if residual is not None:
            residual.append(x)
    return lin(W, "head", rms(x, float(cfg["norm"]["eps"])) * W["final.norm"])


def greedy(W, cfg, prompt, count: int) -> List[int]:
    toks = list(prompt)
    for _ in range(count):
        toks.append(int(forward(W, cfg, toks)[-1].argmax()))
    return toks[len(prompt):]


# ---- tensors ------------------------------------------------------------------------------------
def tensor_shapes(cfg) -> Dict[str, tuple]:
    """Every tensor a model folder of this design holds, with its shape."""
    Wd, vocab = int(cfg["width"]), int(cfg["vocab"])
    out = {"embed": (vocab, Wd), "final.norm": (Wd,), "head": (vocab, Wd)}
    for i, L in enumerate(cfg["layers"]):
        p, q, m = f"l{i}.", f"l{i}.mix.", L["mixer"]
        H, D, V = int(m["heads"]), int(m["dim"]), int(m["vdim"])
        out.update({p + "norm1": (Wd,), p + "norm1b": (Wd,), q + "o": (Wd, H * V)})
        if L["type"] == "mlstm":
            out.update({q + "q": (H * D, Wd), q + "k": (H * D, Wd), q + "v": (H * V, Wd), q + "g": (H * V, Wd),
                        q + "norm": (H * V,)})
            for n in "if":
                out.update({q + n: (H, Wd), q + n + ".b": (H,)})
        elif L["type"] == "latent_attention":
            E, R = int(m["rot_dim"]), int(m["kv_rank"])
            out.update({q + "q": (H * (D + E), Wd), q + "dkv": (R + E, Wd), q + "dkv.norm": (R,), q + "uk": (H * D, R),
                        q + "uv": (H * V, R)})
        else:
            G = int(m["kv_heads"])
            rows = {"q": H * D} if m.get("kv_from") is not None else {"q": H * D, "k": G * D, "v": G * V}
            for n, size in rows.items():
                out.update({q + n: (size, Wd), q + n + ".b": (size,)})
        if L.get("mlp") is not None:
            out.update({p + "norm2": (Wd,), p + "norm2b": (Wd,)})
            q, mlp = p + "mlp.", L["mlp"]
            N, F = int(mlp["router"]["experts"]), int(mlp["expert"]["ff"])
            out[q + "router"] = (N, Wd)
            for e in range(N):
                out.update({q + f"e{e}.up": (F, Wd), q + f"e{e}.down": (Wd, F)})
            if mlp.get("shared"):
                S = int(mlp["shared"]["ff"])
                out.update({q + "shared.up": (S, Wd), q + "shared.down": (Wd, S)})
    return out


def random_tensors(cfg, seed: int) -> Dict[str, torch.Tensor]:
    """Weights with which every mechanism shows in the logits: matrices of unit gain, norm weights around 1, input gates
    around 1 and forget gates that neither die at once nor keep everything.  Rounded to bfloat16, so that a 16-bit
    checkpoint of them is exact."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        tail = name.rsplit(".", 1)[-1]
        if tail.startswith("norm"):
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif name.endswith(".mix.f.b"):
            t = 2.0 + torch.randn(shape, generator=g)
        elif tail == "b":
            t = 0.3 * torch.randn(shape, generator=g)
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        elif name.endswith(".mix.q") or name.endswith(".mix.k"):
            t = 1.5 * torch.randn(shape, generator=g) / shape[-1] ** 0.5
        else:
            t = torch.randn(shape, generator=g) / shape[-1] ** 0.5
        out[name] = t.to(torch.bfloat16).to(F64)
    return out
