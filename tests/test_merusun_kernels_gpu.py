"""Each mechanism of the Merusun decoder alone, kernel against the plain implementation, with inputs made so that a fault
shows: gates that differ by many orders of magnitude, a first token that is still read hundreds of tokens on, memories
carried over portions and slots that change hands; one key whose score stands out at a window's edge and at page borders
for readers with windows of their own; groups whose best expert decides; experts without a gate."""
import math

import pytest
import torch

import plain_merusun as plain

pytestmark = pytest.mark.gpu
DEV = "cuda"
F64 = torch.float64


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def close(got, want, tol, what):
    got, want = got.double().cpu(), want.double()
    err = float((got - want).abs().max() / want.abs().max().clamp(min=1e-30))
    assert torch.isfinite(got).all() and err <= tol, (what, err)


# ---- matrix memory ------------------------------------------------------------------------------
class Memory:
    """One layer's matrix memory on the device: steps of portions of several sequences over shared slots."""

    def __init__(self, H, D, V, cap, blocks, slots=2):
        from allpaca_b200.parts import Workspace
        self.sizes, self.cap = (H, D, V), cap
        self.ws = Workspace(torch.device(DEV)) if blocks else None
        floats = H * D * (V + 1)
        self.rows = torch.full((slots, floats + H + 3), float("nan"), device=DEV)     # a slot holds more than this layer's
        self.state = self.rows[:, :floats].unflatten(1, (H, D, V + 1))
        self.top = self.rows[:, floats:floats + H]

    def step(self, parts):
        """parts: (tensors by name, first position, slot) per sequence; the read-outs over their denominators."""
        from allpaca_b200 import ops
        H, D, V = self.sizes
        cat = {n: torch.cat([p[0][n] for p in parts]).to(DEV).contiguous() for n in parts[0][0]}
        starts = [0]
        for p in parts:
            starts.append(starts[-1] + p[0]["q"].shape[0])
        T = starts[-1]
        place = (i32(starts), i32([p[1] + i for p in parts for i in range(p[0]["q"].shape[0])]), i32([p[2] for p in parts]))
        gates = torch.cat([torch.full((T, 2), float("nan"), device=DEV), cat["i"], cat["f"]], dim=1)
        gi, gf = gates[:, 2:2 + H], gates[:, 2 + H:]
        floor = torch.full((T, H), float("nan"), device=DEV)
        ops.exp_gates(gi, gf, cat["bi"][0].contiguous(), cat["bf"][0].contiguous(), self.cap, self.top, *place, floor, len(parts))
        y = torch.full((T, H * (V + 1)), float("nan"), device=DEV)
        ops.linear_scan(cat["q"], cat["k"], cat["v"], y, self.state, *place, len(parts), H, H, D, V, "head_ready",
                        decay_head=gf, write_gate=gi, unit_column=True, out_scale=D ** -0.5, workspace=self.ws)
        y = y.double().cpu().reshape(T, H, V + 1)
        below = torch.maximum(y[..., V].abs(), floor.double().cpu()) + plain.READ_EPS
        out = (y[..., :V] / below[..., None]).reshape(T, H * V)
        return [out[starts[j]:starts[j + 1]] for j in range(len(parts))]


def draw(H, D, V, n, g, spread=2.0):
    bi, bf = torch.randn(H, generator=g), 2.0 + torch.randn(H, generator=g)
    return {"q": torch.randn(n, H * D, generator=g), "k": torch.randn(n, H * D, generator=g),
            "v": torch.randn(n, H * V, generator=g), "i": spread * torch.randn(n, H, generator=g),
            "f": spread * torch.randn(n, H, generator=g), "bi": bi.repeat(n, 1), "bf": bf.repeat(n, 1)}


def plain_read(t, H, D, V, cap):
    t = {k: v.double() for k, v in t.items()}
    n = t["q"].shape[0]
    i = plain.capped(t["i"] + t["bi"], cap)
    f = torch.nn.functional.logsigmoid(plain.capped(t["f"] + t["bf"], cap))
    q, k, v = (t[x].reshape(n, H, -1) for x in "qkv")
    return plain.matrix_memory(q * D ** -0.5, k, v, i, f).reshape(n, H * V)


def cut(t, a, b):
    return {n: x[a:b] for n, x in t.items()}


def read_error(got, want, what, tol=5e-5):
    """A denominator near its floor or a cancelling product makes single read-outs large: rows are judged by their own size."""
    assert torch.isfinite(got).all(), what
    err = (got - want).abs().max(-1).values / want.abs().max(-1).values.clamp(min=0.05)
    assert float(err.max()) <= tol, (what, int(err.argmax()), float(err.max()))


@pytest.mark.parametrize("blocks", [False, True])
@pytest.mark.parametrize("H,D,V,cap", [(3, 20, 24, 4.0), (1, 136, 40, 15.0), (4, 16, 64, 0.75), (5, 3, 1, 2.0), (2, 6, 10, 30.0),
                                       (2, 7, 3, 5.0), (1, 1, 1, 1.0), (8, 128, 128, 15.0), (2, 256, 100, 10.0)])
def test_memories_over_portions_and_slots(H, D, V, cap, blocks):
    """Two sequences whose portions share steps (a single row beside a long portion, portions of two rows, portions that
    end inside a block of eight), on slots that held something else before; then a slot that changes hands."""
    g = torch.Generator().manual_seed(H * 10 + D)
    run = Memory(H, D, V, cap, blocks)
    ta, tb = draw(H, D, V, 61, g), draw(H, D, V, 9, g)
    ta["bi"][:], ta["bf"][:] = tb["bi"][0], tb["bf"][0]
    ya, yb = [], []
    r = run.step([(cut(ta, 0, 17), 0, 1), (cut(tb, 0, 1), 0, 0)]); ya.append(r[0]); yb.append(r[1])
    r = run.step([(cut(tb, 1, 3), 1, 0), (cut(ta, 17, 18), 17, 1)]); yb.append(r[0]); ya.append(r[1])
    r = run.step([(cut(ta, 18, 41), 18, 1), (cut(tb, 3, 9), 3, 0)]); ya.append(r[0]); yb.append(r[1])
    for a, b in ((41, 43), (43, 51), (51, 54), (54, 61)):
        ya += run.step([(cut(ta, a, b), a, 1)])
    read_error(torch.cat(ya), plain_read(ta, H, D, V, cap), "long sequence", 2e-4)
    read_error(torch.cat(yb), plain_read(tb, H, D, V, cap), "short sequence", 2e-4)
    tc = draw(H, D, V, 5, g)
    read_error(run.step([(tc, 0, 1)])[0], plain_read(tc, H, D, V, cap), "in a slot used before", 2e-4)


@pytest.mark.parametrize("sizes", [[1, 3000, 2], [1024], [1023, 1, 1025], [33, 700]])
def test_running_maximum_along_long_portions(sizes):
    """The two gates and the floor of every token, and the maximum a slot is left with, against a walk token by token:
    portions longer than a CTA takes at a time, gates that now and then leap, a request that goes on from its slot."""
    from allpaca_b200 import ops
    H, cap = 3, 12.0
    g = torch.Generator().manual_seed(sum(sizes))
    T = sum(sizes)
    raw_i, raw_f = 3 * torch.randn(T, H, generator=g), 4.0 + 3 * torch.randn(T, H, generator=g)
    raw_i[torch.rand(T, H, generator=g) < 0.01] = 40.0
    raw_f[torch.rand(T, H, generator=g) < 0.01] = -40.0
    bi, bf = torch.randn(H, generator=g), torch.randn(H, generator=g)
    starts, positions = [0], []
    for j, n in enumerate(sizes):
        starts.append(starts[-1] + n)
        first = 0 if j % 2 == 0 else 7
        positions += range(first, first + n)
    state = torch.randn(len(sizes) + 1, H + 2, generator=g)
    slots = list(range(len(sizes), 0, -1))
    dev = state.to(DEV)
    gi, gf, floor = raw_i.to(DEV), raw_f.to(DEV), torch.empty(T, H, device=DEV)
    ops.exp_gates(gi, gf, bi.to(DEV), bf.to(DEV), cap, dev[:, :H], i32(starts), i32(positions), i32(slots), floor, len(sizes))
    i = plain.capped(raw_i.double() + bi.double(), cap)
    f = torch.nn.functional.logsigmoid(plain.capped(raw_f.double() + bf.double(), cap))
    for j, n in enumerate(sizes):
        top = torch.zeros(H, dtype=F64) if j % 2 == 0 else state[slots[j], :H].double()
        for t in range(starts[j], starts[j + 1]):
            new = torch.maximum(f[t] + top, i[t])
            want = torch.stack([torch.exp(f[t] + top - new), torch.exp(i[t] - new), torch.exp(-new)])
            got = torch.stack([gf[t], gi[t], floor[t]]).double().cpu() if t % 97 == 0 or n < 40 or t - starts[j] in (1023, 1024) else None
            if got is not None:
                assert float(((got - want).abs() / want.clamp(min=1e-12)).max()) <= 2e-4, (j, t, got, want)
            top = new
        close(dev[slots[j], :H], top, 1e-5, ("maximum left in the slot", j))
    assert torch.equal(dev[:, H:].cpu(), state[:, H:]) and torch.equal(dev[0].cpu(), state[0])


@pytest.mark.parametrize("blocks", [False, True])
def test_the_first_token_is_read_hundreds_of_tokens_on(blocks):
    """Every token writes its value along a key of its own kind; the first is written so strongly (its log gate is the
    cap) that everything after it stays small beside it, and nothing is forgotten: rows late in many portions still read
    it, in the numerator and in the denominator."""
    D, V, n, cap = 4, 3, 300, 15.0
    g = torch.Generator().manual_seed(2)
    t = draw(1, D, V, n, g)
    t["bi"][:], t["bf"][:] = 0.0, 0.0
    t["i"][:] = -3.0
    t["i"][0] = 200.0                                  # cap * tanh: 15
    t["f"][:] = 200.0                                  # log gate of -3e-7
    t["k"][:] = torch.tensor([0.0, 1.0, 0.0, 0.0])
    t["k"][0] = torch.tensor([1.0, 0.0, 0.0, 0.0])
    t["q"][:] = torch.tensor([0.0, 1.0, 0.0, 0.0])
    t["q"][150] = t["q"][-1] = t["k"][0]
    run = Memory(1, D, V, cap, blocks, slots=1)
    got, at = [], 0
    for m in [1, 2, 64, 1, 1, 33, 2, 100, 96]:
        got += run.step([(cut(t, at, at + m), at, 0)])
        at += m
    assert at == n
    got = torch.cat(got)
    # along its own key the first value reads back as itself (but for the 1e-6 on the denominator under the scale)
    for row in (150, 299):
        close(got[row], t["v"][0].double(), 1e-4, ("the first token's value", row))
    read_error(got[1:], plain_read(t, 1, D, V, cap)[1:], "all rows", 1e-3)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,V", [(3, 8), (6, 80), (1, 300), (4, 1), (2, 257), (16, 128)])
def test_read_out_over_its_denominator_normed_and_gated(dtype, H, V):
    """An eps of the size of the read-outs, so that the denominators count; some are held up by the floor."""
    from allpaca_b200 import ops
    g = torch.Generator().manual_seed(V)
    T = 37
    y, gate = torch.randn(T, H * (V + 1) + 3, generator=g) * 5, torch.randn(T, 2 * H * V, generator=g)
    floor, w = torch.exp(torch.randn(T, H, generator=g)) * 3, 1 + 0.3 * torch.randn(H * V, generator=g)
    out = torch.empty(T, H * V, dtype=dtype, device=DEV)
    ops.head_norm_gate(y.to(DEV)[:, :H * (V + 1)], gate.to(DEV)[:, H * V:], w.to(DEV), 0.5, out, H, V, activation="sigmoid",
                       floor=floor.to(DEV), floor_eps=0.25)
    z = y[:, :H * (V + 1)].double().reshape(T, H, V + 1)
    o = z[..., :V] / (torch.maximum(z[..., V].abs(), floor.double()) + 0.25)[..., None]
    want = plain.rms(o, 0.5).reshape(T, H * V) * w.double() * torch.sigmoid(gate[:, H * V:].double())
    close(out, want, 1e-5 if dtype == torch.float32 else 1e-2, "read-out")


# ---- attention ----------------------------------------------------------------------------------
def paged(rows, P, order, first_live):
    """rows [T, G, F] of one sequence -> its pages by number and its table row; pages wholly before ``first_live`` were given
    back (NaN, table entry -1)."""
    T, G, F = rows.shape
    pages, table = {}, []
    for b in range(-(-T // P)):
        page = torch.full((G, P, F), float("nan"))
        live = (b + 1) * P > first_live
        if live:
            part = rows[b * P:(b + 1) * P]
            page[:, :part.shape[0]] = part.transpose(0, 1)
            page[:, part.shape[0]:] = 0.0
        pages[order[b]] = page
        table.append(order[b] if live else -1)
    return pages, table


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("H,G,D,E,P,windows", [(6, 3, 24, 40, 8, (21, 37, 9)), (4, 2, 80, 64, 16, (70, 100, 1)),
                                               (3, 1, 20, 12, 8, (11, 12)), (8, 2, 128, 128, 32, (300, 40))])
def test_readers_of_one_layers_keys_behind_windows_of_their_own(dtype, tol, H, G, D, E, P, windows):
    """A layer stores unit-mean-square keys and its values; it and later layers read them with queries and windows of
    their own, one in the softmax's denominator.  A portion of 37 rows behind 300 cached tokens and a single row at
    position 333; for chosen rows the oldest key the reader's window shows dominates, or the one just behind it, or a page's
    last slot.  Pages that no reader sees any more are gone."""
    from allpaca_b200 import ops
    g = torch.Generator().manual_seed(H * 100 + D)
    lens, eps = [(300, 37), (333, 1)], 1e-5
    scale = 4.0 / math.sqrt(D) / math.sqrt(D)
    zero = torch.zeros(H, device=DEV)
    base, store, tables, kv = 0, {}, [], []
    for before, now in lens:
        T = before + now
        k, v = plain.rms(torch.randn(T, G, D, generator=g).double(), eps), torch.randn(T, G, E, generator=g)
        k, v = k.to(dtype).double(), v.to(dtype).double()
        kv.append((k, v))
        n = -(-T // P)
        pages, table = paged(torch.cat([k, v], dim=-1).float(), P, [base + n - 1 - b for b in range(n)], before - max(windows) + 1)
        store.update(pages)
        tables.append(table)
        base += n
    pages = torch.stack([store[b] for b in range(base)]).to(dtype).to(DEV)
    width = max(len(r) for r in tables)
    bt = i32([r + [-1] * (width - len(r)) for r in tables])
    positions = i32([p for before, now in lens for p in range(before, before + now)])
    seq = i32([0] * 37 + [1])
    for w in windows:
        raw, want = [], []
        for (before, now), (k, v) in zip(lens, kv):
            T = before + now
            q = torch.randn(T, H, D, generator=g)
            spikes = {T - 1: T - w, T - 2: T - 2 - w, before: before - w + 1, before + 1: before + 1 - w,
                      T - 3: (T - 3 - w + P) // P * P - 1, T - 4: T - 4}
            for row, key in spikes.items():
                if before <= row < T and 0 <= key <= row:
                    q[row] = 0.3 * q[row] + 6.0 * k[key].float().repeat_interleave(H // G, dim=0)
            raw.append(q[before:])
            q = plain.rms((q + 0.25).double(), eps).to(dtype).double()
            want.append(plain.attend(q * 1.0, k, v, scale * math.sqrt(D), w, True)[before:])
        raw = torch.cat(raw).reshape(-1, H * D).to(DEV).contiguous()
        q = torch.empty(38, H * D, dtype=dtype, device=DEV)
        # a reader's projection and bias hold queries only
        ops.qk_norm_store(raw, q, None, positions, seq, bt, H, G, D, E, eps, bias=torch.full((H * D,), 0.25, device=DEV))
        for single in (False, True):
            out = torch.empty(38, H * E, dtype=dtype, device=DEV)
            ops.attention_window_bias(q, out, pages, bt, i32([0, 37, 38]), positions, 2, H, G, D, E, scale * math.sqrt(D), w,
                                      bias=None, single_rows=single, sink=zero)
            close(out.float().reshape(-1, H, E), torch.cat(want), tol, ("window", w, single))


@pytest.mark.parametrize("H,R,E,P,window", [(7, 72, 24, 16, 45), (5, 32, 8, 8, 19), (4, 128, 24, 16, 33), (16, 512, 64, 32, 500),
                                            (3, 18, 6, 8, 11), (2, 62, 2, 64, 1)])
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-5), (torch.bfloat16, 2e-2)])
def test_records_of_a_latent_and_a_rotated_part_behind_a_window(dtype, tol, H, R, E, P, window):
    """Attention in the latent space, an ordinary softmax: a record is the latent (which is also the value) and the rotated
    part.  A portion of 29 rows behind 500 tokens and a single row of another sequence; one head looks hard at the oldest
    record the window shows, another at the one behind it, one at a page's first slot."""
    from allpaca_b200 import ops
    from allpaca_b200.parts import Workspace
    g = torch.Generator().manual_seed(H + R)
    lens, rec, scale = [(500, 29), (610, 1)], R + E, 1.0 / math.sqrt(R + E)
    base, store, tables, qs, want = 0, {}, [], [], []
    for before, now in lens:
        T = before + now
        r = torch.randn(T, rec, generator=g).to(dtype).double()
        q = torch.randn(T, H, rec, generator=g)
        for n, (row, key) in enumerate({T - 1: T - window, T - 2: T - 2 - window, before: before - window + 1, before + 1: before + 1 - window,
                                        T - 3: (T - 3) // P * P, T - 4: (T - 4 - window + P) // P * P}.items()):
            if before <= row < T and 0 <= key <= row:
                q[row, n % H] = 6.0 * math.sqrt(rec) * r[key].float() / r[key].norm()
        for h, key in enumerate((T - window, T - window - 1)[:H] if now == 1 else ()):
            if key >= 0:
                q[T - 1, h] = 6.0 * math.sqrt(rec) * r[key].float() / r[key].norm()
        q = q.to(dtype).double()
        want.append(plain.attend(q, r[:, None], r[:, None, :R], scale, window, False)[before:])
        qs.append(q[before:])
        n = -(-T // P)
        pages, table = paged(r[:, None].float(), P, [base + n - 1 - b for b in range(n)], before - window + 1)
        store.update(pages)
        tables.append(table)
        base += n
    pages = torch.stack([store[b] for b in range(base)]).to(dtype).to(DEV)[:, 0].contiguous()
    width = max(len(x) for x in tables)
    bt = i32([x + [-1] * (width - len(x)) for x in tables])
    positions = i32([p for before, now in lens for p in range(before, before + now)])
    q = torch.cat(qs).reshape(-1, H * rec).to(dtype).to(DEV).contiguous()
    out = torch.full((30, H * R), float("nan"), dtype=dtype, device=DEV)
    ops.attention_window_bias(q, out, pages, bt, i32([0, 29, 30]), positions, 2, H, 1, rec, R, scale, window, None, None,
                              single_rows=False, other_rows=True, bias=None, record=rec, value_offset=0)
    close(out.float().reshape(-1, H, R), torch.cat(want), tol, "general kernel")
    if dtype == torch.bfloat16 and ops.latent_decode_takes(rec, R):
        for context in (1, 4096):
            one = torch.full((30, H * R), float("nan"), dtype=dtype, device=DEV)
            ops.latent_decode(q, one, pages, bt, i32([0, 29, 30]), positions, 2, H, rec, R, scale, None, context,
                              Workspace(torch.device(DEV)), window=window)
            close(one[29:].float().reshape(-1, H, R), want[1], tol, ("decode kernel", context))


# ---- routed experts -----------------------------------------------------------------------------
@pytest.mark.parametrize("E,top,count,keep", [(14, 3, 2, 1), (10, 3, 5, 2), (256, 16, 8, 3), (9, 2, 9, 2), (64, 1, 1, 1),
                                              (33, 5, 3, 3), (6, 2, 3, 1), (200, 7, 40, 4), (128, 8, 128, 8), (1, 1, 1, 1)])
@pytest.mark.parametrize("T", [3, 600])
def test_choice_among_the_best_groups(E, top, count, keep, T):
    """Experts, shares and groups of every row against the plain routing; row 0's best expert stands alone in a group of
    weak ones, so that it drags them in and keeps the second best group's strong ones out."""
    from allpaca_b200 import ops
    g = torch.Generator().manual_seed(E + T)
    K, scale = 48, 1.75
    rows, router = torch.randn(T, K, generator=g), torch.randn(E, K, generator=g)
    z = rows.double() @ router.double().T
    if E // count > 1 and count > 1:
        want_z = -5.0 + 0.01 * torch.arange(E, dtype=F64)
        want_z[0] = 4.0
        want_z[E // count:2 * (E // count)] += 8.5
        if E <= K:
            rows[0] = torch.linalg.lstsq(router.double(), want_z[:, None]).solution[:, 0].float()
            z = rows.double() @ router.double().T
    r = {"top": top, "scale": scale, "groups": {"count": count, "keep": keep}}
    want, share = plain.route(z, r)
    chosen = torch.empty(T, top, dtype=torch.int32, device=DEV)
    weight = torch.empty(T, top, device=DEV)
    ops.moe_route_rows(rows.to(DEV), router.to(DEV), None, chosen, weight, "softmax_scores", groups=count, keep=keep, scale=scale)
    # two logits a rounding apart may change places: such rows are rare and left out
    gap = torch.sort(z, dim=-1).values.diff(dim=-1).min(-1).values if E > 1 else torch.ones(T)
    sure = gap > 1e-5
    assert float(sure.double().mean()) > 0.5
    assert torch.equal(chosen.cpu().long()[sure], want[sure])
    close(weight.cpu()[sure], share[sure], 1e-5, "shares")


@pytest.mark.parametrize("mode", ["top_softmax", "softmax_all", "sigmoid", "softmax_scores"])
def test_groups_and_scale_with_every_kind_of_routing(mode):
    """With a bias that steers the choice: the groups are ordered by what the choice goes by, and the shares do not see it."""
    from allpaca_b200 import ops
    g = torch.Generator().manual_seed(7)
    T, E, K, top, count, keep = 90, 24, 40, 3, 6, 2
    rows, router, bias = torch.randn(T, K, generator=g) * 0.3, torch.randn(E, K, generator=g), torch.randn(E, generator=g) * 0.3
    z = rows.double() @ router.double().T
    s = torch.sigmoid(z) if mode == "sigmoid" else torch.softmax(z, dim=-1)
    key = (z if mode == "top_softmax" else s) + bias.double()
    best = key.reshape(T, count, -1).max(-1).values.topk(keep, dim=-1).indices
    open_to = torch.zeros(T, count, dtype=torch.bool).scatter(1, best, True).repeat_interleave(E // count, dim=1)
    want = key.masked_fill(~open_to, -math.inf).topk(top, dim=-1).indices
    share = s.gather(1, want)
    if mode == "top_softmax":
        share = torch.softmax(key.gather(1, want), dim=-1)
    elif mode == "softmax_all":
        share = share / share.sum(-1, keepdim=True)
    chosen, weight = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
    ops.moe_route_rows(rows.to(DEV), router.to(DEV), bias.to(DEV), chosen, weight, mode, groups=count, keep=keep, scale=0.5)
    assert torch.equal(chosen.cpu().long(), want)
    close(weight, 0.5 * share, 1e-5, "shares")


def test_logits_that_are_no_numbers_choose_within_the_experts():
    from allpaca_b200 import ops
    rows, router = torch.full((4, 16), float("nan"), device=DEV), torch.ones(6, 16, device=DEV)
    chosen, weight = torch.full((4, 2), 77, dtype=torch.int32, device=DEV), torch.empty(4, 2, device=DEV)
    for groups, keep in ((1, 1), (3, 1)):
        ops.moe_route_rows(rows, router, None, chosen, weight, "softmax_scores", groups=groups, keep=keep)
        assert int(chosen.min()) >= 0 and int(chosen.max()) < 6


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("W,F,E,top,count,keep,shared,T", [(72, 40, 6, 2, 3, 2, 24, 150), (128, 64, 9, 3, 1, 1, 64, 5),
                                                           (40, 24, 5, 1, 5, 1, None, 70), (64, 96, 4, 4, 2, 2, 8, 1),
                                                           (128, 32, 12, 6, 4, 2, 48, 700), (42, 7, 3, 2, 1, 1, 5, 33)])
def test_experts_without_a_gate_and_a_shared_one(dtype, tol, W, F, E, top, count, keep, shared, T):
    from allpaca_b200.parts import BuildEnv, PartSpec, Workspace, build
    g = torch.Generator().manual_seed(W + E)
    w = {"router": torch.randn(E, W, generator=g) * 0.3}
    for n, f in [(f"e{e}", F) for e in range(E)] + ([("shared", shared)] if shared else []):
        w.update({n + ".up": torch.randn(f, W, generator=g) * 0.25, n + ".down": torch.randn(W, f, generator=g) * 0.2})
    w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
    h = torch.randn(T, W, generator=g).to(dtype)
    if dtype == torch.bfloat16:
        top, keep = E, count                             # rounding may swap two experts with close scores: choose all
    groups = {"count": count, "keep": keep}
    dev = torch.device(DEV)
    part = build("feed_forward", PartSpec("routed_experts", {
        "hidden_size": W, "expert_size": F, "experts": E, "top": top, "activation": "relu2", "gated": False,
        "routing": "softmax_scores", "router_bias": False, "groups": groups, "share_scale": 1.6,
        "shared": {"size": shared} if shared else None}), BuildEnv(dtype, dev, Workspace(dev)))
    part.load({k: v.to(dtype).to(dev) for k, v in w.items()})

    class Step:
        max_query_len = T
    got = part.forward(h.to(DEV), Step()).sum(0)
    mlp = {"router": {"experts": E, "top": top, "scale": 1.6, "groups": groups}, "expert": {"ff": F}}
    if shared:
        mlp["shared"] = {"ff": shared}
    close(got, plain.experts({"x." + k: v.double() for k, v in w.items()}, "x.", mlp, h.double()), tol, "routed feed-forward")


@pytest.mark.parametrize("M,N,K", [(1, 40, 64), (8, 1024, 2048), (37, 200, 96), (64, 128, 4096), (100, 96, 320), (200, 256, 512),
                                   (300, 1024, 256), (700, 136, 128), (2048, 1024, 512), (520, 4096, 6400)])
@pytest.mark.parametrize("out_dtype", [torch.bfloat16, torch.float32])
def test_squared_relu_in_the_products_epilogue(M, N, K, out_dtype):
    """Whatever kernel the shape is given to: slices of K in a cluster, one tile to a CTA, persistent, pairs of SMs."""
    from allpaca_b200 import ops
    from allpaca_b200.parts.linear import Linear
    g = torch.Generator().manual_seed(M + N)
    a, w = torch.randn(M, K, generator=g).to(torch.bfloat16), (torch.randn(N, K, generator=g) * K ** -0.5).to(torch.bfloat16)
    z = torch.relu(a.double() @ w.double().T)
    ad, wd = a.to(DEV), w.to(DEV)
    out = torch.full((M, N), float("nan"), dtype=out_dtype, device=DEV)
    Linear.tensor_core_product(ad, wd, out, activation="relu2")
    tol = 3e-5 if out_dtype == torch.float32 else 1e-2
    close(out, z * z, tol, "the kernel of the shape")
    if M > 64:
        for product in (ops.gemm_tc_persistent, ops.gemm_tc_pair):
            out.fill_(float("nan"))
            product(ad, wd, out, activation="relu2")
            close(out, z * z, tol, product.__name__)
    ops.check_kernel_status()


@pytest.mark.parametrize("W", [64, 42, 320, 2048, 4100, 8192, 20000])
@pytest.mark.parametrize("T", [3, 700])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_one_stream_between_two_norms(W, T, dtype):
    """A sublayer's normed result into the stream and the norm of what the next one reads, in steps of few rows and many;
    chosen rows leave the stream alone."""
    from allpaca_b200 import ops
    g = torch.Generator().manual_seed(W + T)
    x, d = torch.randn(T, 1, W, generator=g), 5 * torch.randn(1, T, W, generator=g)
    w, sw = 1 + 0.2 * torch.randn(W, generator=g), torch.randn(1, W, generator=g)
    one = torch.ones(1, device=DEV)
    want = x.double()[:, 0] + plain.rms(d.double()[0], 0.3) * sw.double()
    read = plain.rms(want, 1e-5) * w.double()
    kw = dict(delta=d.to(DEV), out_w=one, mix=one.view(1, 1), slice_weight=sw.to(DEV), slice_eps=0.3)
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    xd, out = x.to(DEV), torch.empty(T, W, dtype=dtype, device=DEV)
    ops.stream_norm(xd, one, w.to(DEV), 1e-5, out, **kw)
    close(xd[:, 0], want, 2e-5, "the stream")
    close(out, read, tol, "what the sublayer reads")
    xd, out = x.to(DEV), torch.empty(2, W, dtype=dtype, device=DEV)
    ops.stream_norm(xd, one, w.to(DEV), 1e-5, out, rows=i32([T - 1, 0]), **kw)
    close(out, read[[T - 1, 0]], tol, "chosen rows")
    assert torch.equal(xd.cpu(), x)
