"""Each mechanism of the Boketar decoder alone, kernel against the plain implementation, with inputs made so that a fault
shows: one key whose score stands out (far back, at page borders, the oldest the window shows, the one behind it) beside
sinks that weigh as much as the keys; neighbouring pairs rotated at far positions behind a convolution whose inputs lie in
the request's state; recurrences carried over portions and slots that change hands, token after token and eight tokens at a
time; decays that forget nothing, and ones that forget at once; streams that mix; two results normed apart."""
import math

import pytest
import torch

import plain_boketar as plain

pytestmark = pytest.mark.gpu
DEV = "cuda"
F64 = torch.float64


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def close(got, want, tol, what):
    got, want = got.double().cpu(), want.double()
    err = float((got - want).abs().max() / want.abs().max().clamp(min=1e-30))
    assert torch.isfinite(got).all() and err <= tol, (what, err)


def paged(kv, P, order, first_live):
    """kv [T, G, F] of one sequence -> its pages by number and its table row; pages wholly before ``first_live`` were given
    back (NaN, table entry -1)."""
    T, G, F = kv.shape
    pages, table = {}, []
    for b in range(-(-T // P)):
        page = torch.full((G, P, F), float("nan"))
        live = (b + 1) * P > first_live
        if live:
            rows = kv[b * P:(b + 1) * P]
            page[:, :rows.shape[0]] = rows.transpose(0, 1)
            page[:, rows.shape[0]:] = 0.0
        pages[order[b]] = page
        table.append(order[b] if live else -1)
    return pages, table


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("H,G,D,E,P,window", [(6, 3, 24, 40, 8, 21), (2, 1, 64, 64, 16, 72), (8, 2, 80, 48, 16, 120),
                                              (3, 3, 136, 16, 16, 1), (4, 1, 20, 12, 8, 11), (12, 4, 192, 128, 32, 300)])
def test_window_and_sink_with_a_key_that_stands_out(dtype, tol, H, G, D, E, P, window):
    """Two sequences in one launch: a portion of 37 rows behind 300 cached tokens and a single decoded row at position 333
    of another.  In each, one key is made to dominate for chosen rows: the oldest the window still shows, the one just
    behind it, a page's first and last slot.  One head's sink outweighs every key, one weighs nothing."""
    from allpaca_b200 import ops
    g = torch.Generator().manual_seed(H * 100 + D)
    lens = [(300, 37), (333, 1)]                       # (cached before, rows now)
    scale = 1.0 / math.sqrt(D)
    sink = 1.0 + torch.randn(H, generator=g)
    sink[0], sink[-1] = 12.0, -40.0
    qs, store, tables, want, base = [], {}, [], [], 0
    for before, now in lens:
        T = before + now
        q, k, v = (torch.randn(T, n, d, generator=g) for n, d in ((H, D), (G, D), (G, E)))
        w = window
        spikes = {T - 1: T - w, T - 2: T - 2 - w, before: max(0, before - w + 1), before + 1: (before // P) * P,
                  T - 3: ((T - 3 - w + 1 + P - 1) // P) * P + P - 1 if w > 2 * P else T - 3}
        for row, key in spikes.items():
            if 0 <= key <= row < T and row >= before:
                k[key] = 0.3 * k[key] + 4.0 * q[row, ::H // G] / q[row, ::H // G].norm(dim=-1, keepdim=True) * math.sqrt(D)
        q, k, v = (t.to(dtype).float() for t in (q, k, v))
        want.append(plain.attend(q.double(), k.double(), v.double(), scale, w, sink.double())[before:])
        qs.append(q[before:])
        n = -(-T // P)
        pages, table = paged(torch.cat([k, v], dim=-1), P, [base + n - 1 - b for b in range(n)], before - w + 1)
        store.update(pages)
        tables.append(table)
        base += n
    pages = torch.stack([store[b] for b in range(base)]).to(dtype).to(DEV)
    width = max(len(r) for r in tables)
    bt = i32([r + [-1] * (width - len(r)) for r in tables])
    q = torch.cat(qs).reshape(-1, H * D).to(dtype).to(DEV).contiguous()
    positions = i32([p for before, now in lens for p in range(before, before + now)])
    for single in (False, True):                       # the general kernels for all rows; the decode kernel for the single row
        out = torch.empty(q.shape[0], H * E, dtype=dtype, device=DEV)
        ops.attention_window_bias(q, out, pages, bt, i32([0, 37, 38]), positions, 2, H, G, D, E, scale, window,
                                  bias=None, single_rows=single, sink=sink.to(DEV))
        close(out.float().reshape(-1, H, E), torch.cat(want), tol, ("attention", single))


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 2e-2)])
def test_single_rows_over_key_slices_with_a_sink(dtype, tol):
    """A window of 1500 keys: the decode kernel shares a sequence's key tiles between the CTAs of a cluster; the sink counts
    once for all of them.  Beside it a sequence so short that most of them see no key."""
    from allpaca_b200 import ops
    H, G, D, E, P, window = 4, 2, 32, 48, 16, 1500
    g = torch.Generator().manual_seed(5)
    sink = torch.tensor([4.0, 7.0, 2.0, -3.0])
    lens = [2101, 7]
    qs, store, tables, want, base = [], {}, [], [], 0
    for T in lens:
        q, k, v = (torch.randn(T, n, d, generator=g) for n, d in ((H, D), (G, D), (G, E)))
        key = max(0, T - window)
        k[key] = 5.0 * q[T - 1, ::H // G] / q[T - 1, ::H // G].norm(dim=-1, keepdim=True)
        q, k, v = (t.to(dtype).float() for t in (q, k, v))
        lo = max(0, T - window)
        s = torch.stack([q[-1, a].double() @ k[lo:, a // (H // G)].double().T for a in range(H)]) * 0.4
        w = torch.softmax(torch.cat([s, sink.double()[:, None]], dim=1), dim=-1)[:, :-1]
        want.append(torch.stack([w[a] @ v[lo:, a // (H // G)].double() for a in range(H)])[None])
        qs.append(q[-1:])
        n = -(-T // P)
        pages, table = paged(torch.cat([k, v], dim=-1), P, [base + n - 1 - b for b in range(n)], lo)
        store.update(pages)
        tables.append(table)
        base += n
    pages = torch.stack([store[b] for b in range(base)]).to(dtype).to(DEV)
    bt = i32([r + [-1] * (max(map(len, tables)) - len(r)) for r in tables])
    q = torch.cat(qs).reshape(-1, H * D).to(dtype).to(DEV).contiguous()
    out = torch.empty(2, H * E, dtype=dtype, device=DEV)
    ops.attention_window_bias(q, out, pages, bt, i32([0, 1, 2]), i32([n - 1 for n in lens]), 2, H, G, D, E, 0.4, window,
                              bias=None, single_rows=True, other_rows=False, max_context=max(lens), sink=sink.to(DEV))
    close(out.float().reshape(-1, H, E), torch.cat(want), tol, "single rows over key slices")


@pytest.mark.parametrize("taps,C,activation", [(3, 40, None), (1, 12, None), (2, 37, None), (7, 24, None), (4, 64, "silu"),
                                               (11, 9, None), (6, 16, "silu")])
def test_convolution_of_biased_inputs_carried_over_portions(taps, C, activation):
    """The bias belongs to the inputs: what is kept for the next portion has it, and what lies before the start is zero
    WITHOUT it.  Two sequences in alternating portions, shorter than the convolution and longer than a run."""
    from allpaca_b200 import ops
    g = torch.Generator().manual_seed(taps)
    L = [45, 17]
    u = [torch.randn(n, C + 8, generator=g) for n in L]
    w, b = torch.randn(C, taps, generator=g), 2.0 + torch.randn(C, generator=g)
    want = [plain.short_conv(x[:, 4:4 + C].double() + b.double(), w.double()) for x in u]
    if activation:
        want = [plain.silu(x) for x in want]
    state = torch.full((3, max(taps - 1, 1), C), float("nan"), device=DEV)      # slots 2 and 0 are used
    got, at, k = [[], []], [0, 0], 0
    cuts = [1, 2, 1, 5, 3, 1, 20, 7, 2, 30]
    while at[0] < L[0] or at[1] < L[1]:
        seqs = []
        for s in (0, 1):
            n = min(cuts[(k + s) % len(cuts)], L[s] - at[s])
            if n > 0:
                seqs.append((s, at[s], n))
        k += 1
        x = torch.cat([u[s][a:a + n] for s, a, n in seqs]).to(DEV).contiguous()
        starts = [0]
        for _, _, n in seqs:
            starts.append(starts[-1] + n)
        out = torch.empty(starts[-1], C, device=DEV)
        ops.causal_conv(x, 4, w.to(DEV), None, state if taps > 1 else None, i32(starts),
                        i32([a + i for _, a, n in seqs for i in range(n)]), i32([2 if s == 0 else 0 for s, _, _ in seqs]),
                        out, len(seqs), activation=activation, in_bias=b.to(DEV))
        for j, (s, _, n) in enumerate(seqs):
            got[s].append(out[starts[j]:starts[j + 1]].cpu())
            at[s] += n
    for s in (0, 1):
        close(torch.cat(got[s]), want[s], 3e-6, ("convolution", s))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,E,dims", [(4, 2, 24, 40, 8), (3, 1, 20, 12, 20), (2, 2, 80, 16, 2), (1, 1, 256, 32, 130)])
def test_neighbouring_pairs_are_rotated_on_the_way_into_the_page(dtype, H, G, D, E, dims):
    from allpaca_b200 import ops
    g = torch.Generator().manual_seed(D + dims)
    positions = [0, 1, 7, 8, 200, 4097, 15]
    T, P = len(positions), 8
    qkv = torch.randn(T, (H + G) * D + G * E, generator=g)
    rot, pos = {"base": 5000.0, "dims": dims}, torch.tensor(positions)
    q = plain.rotate(qkv[:, :H * D].double().reshape(T, H, D), rot, pos)
    k = plain.rotate(qkv[:, H * D:(H + G) * D].double().reshape(T, G, D), rot, pos)
    v = qkv[:, (H + G) * D:].double().reshape(T, G, E)
    f = torch.tensor([5000.0 ** (-2.0 * i / dims) for i in range(dims // 2)])
    table = torch.empty(T, dims // 2, 2, device=DEV)
    ops.rope_table(i32(positions), f.to(DEV), table, 1.0)
    npages = max(positions) // P + 1
    pages = torch.zeros(npages, G, P, D + E, dtype=dtype, device=DEV)
    q_out = torch.empty(T, H * D, dtype=dtype, device=DEV)
    bt = i32([[(3 * b + 1) % npages for b in range(npages)]])
    ops.qk_norm_store(qkv.to(DEV), q_out, pages, i32(positions), i32([0] * T), bt, H, G, D, E, 0.0, normalise=False,
                      cos_sin=table, pairing=1)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    near = [i for i, p in enumerate(positions) if p < 1000]
    close(q_out.float().reshape(T, H, D)[near], q[near], tol, "queries")
    close(q_out.float().reshape(T, H, D), q, max(tol, 5e-4), "queries at far positions")   # a 32-bit angle of thousands of radians
    for i, p in enumerate(positions):
        rec = pages[(3 * (p // P) + 1) % npages, :, p % P].float().cpu()
        close(rec[:, :D], k[i], max(tol, 5e-4), ("key", p))
        close(rec[:, D:], v[i], tol, ("value", p))


class Recurrence:
    """One layer's recurrence on the device: steps of portions of several sequences over shared slots."""

    def __init__(self, kind, H, G, D, V, consts, blocks, slots=2):
        from allpaca_b200.parts import Workspace
        self.kind, self.sizes, self.consts = kind, (H, G, D, V), consts
        self.ws = Workspace(torch.device(DEV)) if blocks else None
        self.state = torch.full((slots, H, D, V), float("nan"), device=DEV)

    def step(self, parts):
        """parts: (tensors by name, first position, slot) per sequence; the read-outs."""
        from allpaca_b200 import ops
        H, G, D, V = self.sizes
        cat = {n: torch.cat([p[0][n] for p in parts]).to(DEV).contiguous() for n in parts[0][0]}
        starts = [0]
        for p in parts:
            starts.append(starts[-1] + p[0]["q"].shape[0])
        positions = [p[1] + i for p in parts for i in range(p[0]["q"].shape[0])]
        y = torch.empty(starts[-1], H * V, device=DEV)
        c = {n: t.to(DEV) for n, t in self.consts.items()}
        if self.kind == "lightning":
            kw = dict(decay="head", decay_const=c["decay"], qk="silu")
        else:
            kw = dict(decay="channel_token", decay_channel=cat["z"], decay_const=c["A_log"], dt_bias=c["dt_bias"],
                      beta=cat["b"], qk="unit", unit_eps=plain.UNIT_EPS, out_scale=D ** -0.5)
        ops.linear_scan(cat["q"], cat["k"], cat["v"], y, self.state, i32(starts), i32(positions),
                        i32([p[2] for p in parts]), len(parts), H, G, D, V, workspace=self.ws, **kw)
        return [y[starts[j]:starts[j + 1]].cpu() for j in range(len(parts))]


def draw(kind, H, G, D, V, n, g):
    t = {"q": torch.randn(n, G * D, generator=g), "k": torch.randn(n, G * D, generator=g),
         "v": torch.randn(n, H * V, generator=g)}
    if kind == "delta":
        t.update(z=2.0 * torch.randn(n, H * D, generator=g), b=torch.randn(n, H, generator=g))
    return t


def plain_read(kind, t, H, G, D, V, consts):
    n = t["q"].shape[0]
    q, k = t["q"].double().reshape(n, G, D), t["k"].double().reshape(n, G, D)
    v = t["v"].double().reshape(n, H, V)
    if kind == "delta":
        z = torch.nn.functional.softplus(t["z"].double() + consts["dt_bias"].double()).reshape(n, H, D)
        decay = torch.exp(-torch.exp(consts["A_log"].double())[None, :, None] * z)
        return plain.delta_recurrence(plain.unit(q) * D ** -0.5, plain.unit(k), v, decay,
                                      torch.sigmoid(t["b"].double())).reshape(n, H * V)
    q, k, v = plain.silu(q), plain.silu(k), plain.silu(v)
    S, out = torch.zeros(H, D, V, dtype=F64), torch.zeros(n, H, V, dtype=F64)
    for i in range(n):
        S = consts["decay"].double()[:, None, None] * S + k[i][:, :, None] * v[i][:, None, :]
        out[i] = torch.einsum("hdv,hd->hv", S, q[i])
    return out.reshape(n, H * V)


def cut(t, a, b):
    return {n: x[a:b] for n, x in t.items()}


@pytest.mark.parametrize("blocks", [False, True])
@pytest.mark.parametrize("kind,H,G,D,V", [
    ("lightning", 3, 3, 16, 8), ("lightning", 1, 1, 64, 100), ("lightning", 5, 5, 6, 10), ("lightning", 2, 2, 130, 7),
    ("lightning", 32, 32, 128, 64), ("delta", 3, 1, 16, 24), ("delta", 4, 2, 40, 16), ("delta", 2, 1, 136, 40), ("delta", 1, 1, 3, 5),
    ("delta", 2, 2, 7, 6), ("delta", 1, 1, 400, 12), ("delta", 16, 8, 128, 128), ("delta", 1, 1, 1, 1)])
def test_recurrences_over_portions_and_slots(kind, H, G, D, V, blocks):
    """Two sequences whose portions share steps (a single row beside a long portion, portions of two rows, portions that
    end inside a block of eight), on slots that held something else before; then a slot that changes hands."""
    g = torch.Generator().manual_seed(H * 10 + D)
    consts = {"decay": torch.tensor(([0.9, 0.97, 0.995, 1.0, 0.5] * 7)[:H]),
              "A_log": torch.log(0.05 + 1.5 * torch.rand(H, generator=g)), "dt_bias": torch.randn(H * D, generator=g) - 0.5}
    run = Recurrence(kind, H, G, D, V, consts, blocks)
    ta, tb = draw(kind, H, G, D, V, 61, g), draw(kind, H, G, D, V, 9, g)
    ya, yb = [], []
    r = run.step([(cut(ta, 0, 17), 0, 1), (cut(tb, 0, 1), 0, 0)]); ya.append(r[0]); yb.append(r[1])
    r = run.step([(cut(tb, 1, 3), 1, 0), (cut(ta, 17, 18), 17, 1)]); yb.append(r[0]); ya.append(r[1])
    r = run.step([(cut(ta, 18, 41), 18, 1), (cut(tb, 3, 9), 3, 0)]); ya.append(r[0]); yb.append(r[1])
    for a, b in ((41, 43), (43, 51), (51, 54), (54, 61)):
        ya += run.step([(cut(ta, a, b), a, 1)])
    close(torch.cat(ya), plain_read(kind, ta, H, G, D, V, consts), 3e-5, "long sequence")
    close(torch.cat(yb), plain_read(kind, tb, H, G, D, V, consts), 3e-5, "short sequence")
    tc = draw(kind, H, G, D, V, 5, g)
    close(run.step([(tc, 0, 1)])[0], plain_read(kind, tc, H, G, D, V, consts), 3e-5, "in a slot used before")


@pytest.mark.parametrize("blocks", [False, True])
def test_channels_forget_on_their_own(blocks):
    """Every token writes its value along its own key channel under a full gate.  Channels that never forget read their
    value hundreds of tokens on, in portions of many sizes; the channel that forgets at once reads nothing of it."""
    D, V, n = 4, 3, 300
    g = torch.Generator().manual_seed(2)
    k = torch.zeros(n, D)
    k[0, 0] = k[1, 1] = 1.0
    k[2:, 3] = 1.0
    q = torch.zeros(n, D)
    q[2:, 3] = 1.0
    q[-2:] = torch.tensor([[1.0, 0, 0, 0], [0, 1.0, 0, 0]])
    v = torch.randn(n, V, generator=g)
    z = torch.full((n, D), -200.0)                     # softplus 0: these channels keep everything
    z[:, 1] = 300.0                                    # exp(-300) at every token
    t = {"q": q, "k": k, "v": v, "z": z, "b": torch.full((n, 1), 80.0)}
    run = Recurrence("delta", 1, 1, D, V, {"A_log": torch.zeros(1), "dt_bias": torch.zeros(D)}, blocks, slots=1)
    got, at = [], 0
    for m in [1, 2, 64, 1, 1, 33, 2, 100, 96]:
        got += run.step([(cut(t, at, at + m), at, 0)])
        at += m
    assert at == n
    got = torch.cat(got) * D ** 0.5
    close(got[-2], v[0], 1e-5, "the first token's value")
    assert float(got[-1].abs().max()) == 0.0
    close(got[2:-2], v[2:-2], 1e-5, "the value written last")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,V,together", [(3, 8, True), (6, 80, True), (4, 40, False), (1, 300, False), (16, 128, True)])
def test_read_out_norm_over_a_head_or_the_row_and_sigmoid_gate(dtype, H, V, together):
    from allpaca_b200 import ops
    g = torch.Generator().manual_seed(V)
    T = 37
    y, gate = torch.randn(T, H * V + 3, generator=g) * 5, torch.randn(T, 2 * H * V, generator=g)
    y[:, :V] *= 10.0                                   # one head dominates where the heads are normed together
    heads, width = (1, H * V) if together else (H, V)
    w = 1 + 0.3 * torch.randn(width, generator=g)
    out = torch.empty(T, H * V, dtype=dtype, device=DEV)
    ops.head_norm_gate(y.to(DEV)[:, :H * V], gate.to(DEV)[:, H * V:], w.to(DEV), 1e-5, out, heads, width, activation="sigmoid")
    o = plain.rms(y[:, :H * V].double().reshape(T, heads, width), 1e-5) * w.double()
    close(out, o.reshape(T, H * V) * torch.sigmoid(gate[:, H * V:].double()), 1e-5 if dtype == torch.float32 else 1e-2, "read-out")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,W,slices", [(1, 64, 1), (2, 96, 2), (3, 42, 2), (4, 2048, 2), (4, 4096, 1), (5, 128, 2), (6, 2052, 1),
                                        (8, 4096, 2), (17, 40, 1), (4, 5000, 2), (3, 4, 3)])
def test_streams_between_two_sublayers(dtype, n, W, slices):
    """The pending result (plain sums, or slices with biases each normed on its own) into the streams, and the norm of what
    the next sublayer reads; without old streams, with nothing pending, and for chosen rows."""
    from allpaca_b200 import ops
    g = torch.Generator().manual_seed(n * 1000 + W)
    T, eps = 13, 1e-5
    x, d = torch.randn(T, n, W, generator=g), torch.randn(slices, T, W, generator=g) * 3
    win, wout, mix = torch.randn(n, generator=g), torch.randn(n, generator=g), torch.randn(n, n, generator=g)
    w, sb, sw = 1 + 0.2 * torch.randn(W, generator=g), torch.randn(slices, W, generator=g), torch.randn(slices, W, generator=g)
    dev = {k: t.to(DEV).contiguous() for k, t in dict(d=d, win=win, wout=wout, mix=mix, w=w, sb=sb, sw=sw).items()}
    tol = 2e-5 if dtype == torch.float32 else 1e-2

    def reads(xs):
        return plain.rms(plain.gather_streams(xs, win.double()), eps) * w.double()
    for normed in (False, True):
        b = d.double() + sb.double()[:, None]
        y = 0.5 * sum(plain.rms(b[s], 3e-4) * sw[s].double() for s in range(slices)) if normed else d.double().sum(0)
        kw = dict(delta=dev["d"], out_w=dev["wout"])
        if normed:
            kw.update(slice_bias=dev["sb"], slice_weight=dev["sw"], slice_eps=3e-4, slice_scale=0.5)
        want = plain.scatter_streams(x.double(), y, wout.double(), mix.double())
        xd, out = x.to(DEV), torch.empty(T, W, dtype=dtype, device=DEV)
        ops.stream_norm(xd, dev["win"], dev["w"], eps, out, mix=dev["mix"], **kw)
        close(xd, want, 2e-5, ("streams", normed))
        close(out, reads(want), tol, ("what the sublayer reads", normed))
        # chosen rows: the same rows, the streams left alone
        xd, out = x.to(DEV), torch.empty(3, W, dtype=dtype, device=DEV)
        ops.stream_norm(xd, dev["win"], dev["w"], eps, out, mix=dev["mix"], rows=i32([5, 0, 12]), **kw)
        close(out, reads(want)[[5, 0, 12]], tol, ("chosen rows", normed))
        assert torch.equal(xd.cpu(), x)
        # the first reader of a step: the old streams (here NaN) do not enter
        xd, out = torch.full((T, n, W), float("nan"), device=DEV), torch.empty(T, W, dtype=dtype, device=DEV)
        ops.stream_norm(xd, dev["win"], dev["w"], eps, out, **kw)
        close(xd, y[:, None, :] * wout.double()[None, :, None], 2e-5, ("first streams", normed))
        close(out, reads(xd.double().cpu()), tol, ("first read", normed))
    xd, out = x.to(DEV), torch.empty(T, W, dtype=dtype, device=DEV)
    ops.stream_norm(xd, dev["win"], dev["w"], eps, out)
    close(out, reads(x.double()), tol, "nothing pending")
    assert torch.equal(xd.cpu(), x)


def test_a_row_has_the_same_bits_in_any_batch():
    from allpaca_b200 import ops
    g = torch.Generator().manual_seed(1)
    n, W = 4, 256
    x, d = torch.randn(40, n, W, generator=g).to(DEV), torch.randn(2, 40, W, generator=g).to(DEV)
    one, w2, mix = torch.ones(n, device=DEV), torch.ones(2, W, device=DEV), torch.randn(n, n, generator=g).to(DEV)
    kw = dict(out_w=one, mix=mix, slice_weight=w2, slice_eps=1e-6)
    out, alone = torch.empty(40, W, device=DEV), torch.empty(1, W, device=DEV)
    xs = x.clone()
    ops.stream_norm(xs, one, w2[0].contiguous(), 1e-6, out, delta=d, **kw)
    for t in (0, 17, 39):
        xt = x[t:t + 1].clone()
        ops.stream_norm(xt, one, w2[0].contiguous(), 1e-6, alone, delta=d[:, t:t + 1].contiguous(), **kw)
        assert torch.equal(alone[0], out[t]) and torch.equal(xt[0], xs[t])
