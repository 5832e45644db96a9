"""The Merusun decoder without a GPU: configuration, tensor names and shapes against the plain list, what each layer asks
of the cache and of the state slots, refused configurations, the order of the rotated coordinates, and each mechanism of
the plain implementation by hand."""
import copy
import math

import pytest
import torch

import plain_merusun as plain
from merusun_configs import CONFIGS

F64 = torch.float64


def build(config, dtype=torch.float32):
    from allpaca_b200.models import DecoderModel, resolve
    from allpaca_b200.parts import BuildEnv, Workspace
    arch = resolve(config)
    cfg = arch.config_class.from_dict(config)
    dev = torch.device("cpu")
    return cfg, DecoderModel(arch.spec_builder(cfg), BuildEnv(dtype, dev, Workspace(dev), page_size=8, max_seqs=2))


@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_names_and_shapes(name, dtype):
    _, model = build(CONFIGS[name], dtype)
    got = {n: tuple(ws.shape) for n, (ws, _, _) in model.weight_targets().items()}
    assert got == plain.tensor_shapes(CONFIGS[name])


def test_cache_plan_and_state():
    cfg, model = build(CONFIGS["A"])
    plan = model.cache_plan()
    # layer 0's keys and values (3 heads of 24 + 40) stay readable as far back as the longest window that reads them
    assert [(g.need.outer, g.need.inner, g.need.window, g.runs) for g in plan] == \
        [((3,), (64,), 37, [0]), ((), (40,), 19, [3])]
    assert [run.cache_from for run in model.spec.order] == [None, None, 0, None, 0]
    # a matrix of 20 x (24 + 1) and a running maximum per head
    assert model.state_bytes() == [0, 4 * 3 * (20 * 25 + 1), 0, 0, 0]
    assert not model.host_control()
    assert model.spec.streams == 1 and cfg.embedding_scale == 5.0
    config = copy.deepcopy(CONFIGS["A"])
    config["layers"][4]["mixer"]["mask"] = None            # a reader without a window keeps every page
    assert build(config)[1].cache_plan()[0].need.window is None


def test_sizes_left_out_take_their_natural_value():
    from allpaca_b200.config import MerusunConfig
    c = copy.deepcopy(CONFIGS["A"])
    for L in c["layers"]:
        L["mixer"].pop("vdim")
        if L["type"] == "attention":
            L["mixer"].pop("kv_heads")
    c["layers"][1]["mlp"]["router"].pop("scale")
    cfg = MerusunConfig.from_dict(c)
    assert [L.mixer.vdim for L in cfg.layers] == [24, 20, 24, 16, 24]
    assert cfg.layers[0].mixer.kv_heads == 6
    m = cfg.layers[1].mlp
    assert (m.scale, m.groups, m.keep, m.shared_ff) == (1.0, 1, 1, None)


def test_refused_configurations():
    from allpaca_b200.config import ConfigError, MerusunConfig

    def broken(change):
        c = copy.deepcopy(CONFIGS["A"])
        change(c)
        with pytest.raises(ConfigError):
            MerusunConfig.from_dict(c)
    broken(lambda c: c["layers"][0].update(type="mamba"))
    broken(lambda c: c["layers"][0]["mixer"].update(kv_heads=4))                        # 6 heads on 4
    broken(lambda c: c["layers"][0]["mixer"]["mask"].update(size=0))
    broken(lambda c: c["layers"][2]["mixer"].update(kv_from=1))                         # a matrix memory keeps no keys
    broken(lambda c: c["layers"][2]["mixer"].update(kv_from=2))                         # itself
    broken(lambda c: c["layers"][4]["mixer"].update(kv_from=2))                         # which has none of its own
    broken(lambda c: c["layers"][2]["mixer"].update(dim=32))                            # not the keys that are there
    broken(lambda c: c["layers"][3]["mixer"].update(kv_from=0))
    broken(lambda c: c["layers"][3]["mixer"]["rot"].update(dims=7))                     # odd
    broken(lambda c: c["layers"][3]["mixer"]["rot"].update(dims=10))                    # more than the rotated part has
    broken(lambda c: c["layers"][1]["mixer"].update(gate_cap=0.0))
    broken(lambda c: c["layers"][1]["mixer"].pop("dim"))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="dense"))
    broken(lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=3))         # 10 experts
    broken(lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=6))
    broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=5))                     # two groups of two
    broken(lambda c: c["norm"].update(eps=0.0))
    broken(lambda c: c.pop("width"))
    broken(lambda c: c.update(layers=[]))


@pytest.mark.parametrize("rot,dims", [(8, 8), (10, 6), (2, 2)])
def test_neighbouring_pairs_become_half_split_ones_at_load(rot, dims):
    """Latent attention turns coordinate i with i + dims/2; for neighbouring pairs the rows of the matrices that form the
    rotated parts are reordered, queries and the shared key part alike, so that the scores are the same."""
    from allpaca_b200.parts import BuildEnv, PartSpec, Workspace, build as build_part
    H, D, R, V, Wd = 3, 5, 7, 4, 12
    dev = torch.device("cpu")
    part = build_part("mixer", PartSpec("latent_attention", {
        "hidden_size": Wd, "num_heads": H, "head_dim": D, "rot_dim": rot, "value_dim": V, "kv_rank": R, "q_rank": 0,
        "scale": 1.0, "norm_eps": 1e-5, "rope": {"dims": dims, "theta": 30.0, "pairing": "adjacent"}}),
        BuildEnv(torch.float32, dev, Workspace(dev)))
    g = torch.Generator().manual_seed(rot)
    t = {n: torch.randn(ws.shape, generator=g) for n, ws in part.weights().items()}
    part.load(t)
    T = 6
    h, pos = torch.randn(T, Wd, generator=g, dtype=F64), torch.arange(T)
    spec = {"base": 30.0, "dims": dims}

    def half_split(x):
        f = torch.tensor([30.0 ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
        a = pos.to(F64)[:, None] * f
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., :dims // 2], x[..., dims // 2:dims]
        return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)
    down = h @ part.down.weight.double().T
    q = down[:, :H * (D + rot)].reshape(T, H, D + rot)
    k = down[:, H * (D + rot) + R:]
    got = torch.einsum("ihd,jd->hij", half_split(q[..., D:]), half_split(k[:, None])[:, 0])
    q = (h @ t["q"].double().T).reshape(T, H, D + rot)
    k = (h @ t["dkv"].double().T)[:, R:]
    want = torch.einsum("ihd,jd->hij", plain.rotate(q[..., D:], spec, pos), plain.rotate(k[:, None], spec, pos)[:, 0])
    assert torch.allclose(got, want, atol=1e-6)
    assert torch.equal(part.down.weight[:D], t["q"][:D])                # the unrotated part lies as it did


def test_mechanisms_by_hand():
    # one in the denominator: two equal scores of zero weigh a third each; a window of two
    v = torch.tensor([[[3.0]], [[6.0]], [[12.0]]], dtype=F64)
    zero = torch.zeros(3, 1, 1, dtype=F64)
    out = plain.attend(zero, zero, v, 1.0, 2, True)
    assert torch.allclose(out[:, 0, 0], torch.tensor([1.5, 3.0, 6.0], dtype=F64))
    out = plain.attend(zero, zero, v, 1.0, 2, False)
    assert torch.allclose(out[:, 0, 0], torch.tensor([3.0, 4.5, 9.0], dtype=F64))
    # neighbouring coordinates turn together, the rest pass
    r = plain.rotate(torch.tensor([[[1.0, 0.0, 1.0, 0.0, 7.0]]], dtype=F64), {"base": 100.0, "dims": 4}, torch.tensor([2]))
    a = 2 * 100.0 ** -0.5
    assert torch.allclose(r[0, 0], torch.tensor([math.cos(2.0), math.sin(2.0), math.cos(a), math.sin(a), 7.0], dtype=F64))
    # the memory: a weak first write (log gate -2) leaves the running maximum at f + 0 = 0, so that the denominator is 1
    one = torch.ones(2, 1, 1, dtype=F64)
    o = plain.matrix_memory(one, one, torch.tensor([[[5.0]], [[7.0]]], dtype=F64),
                            torch.tensor([[-2.0], [3.0]], dtype=F64), torch.tensor([[0.0], [math.log(0.5)]], dtype=F64))
    assert torch.allclose(o[0, 0, 0], torch.tensor(5 * math.exp(-2.0) / (1 + 1e-6), dtype=F64))
    num, den = 0.5 * math.exp(-2.0) * 5 + math.exp(3.0) * 7, 0.5 * math.exp(-2.0) + math.exp(3.0)
    assert abs(float(o[1, 0, 0]) - num / (den + 1e-6 * math.exp(3.0))) < 1e-9
    # groups of two: the best expert is in the second group, the second best in the first, which is not kept
    z = torch.log(torch.tensor([[0.3, 0.05, 0.4, 0.25]], dtype=F64))
    chosen, w = plain.route(z, {"top": 2, "scale": 2.0, "groups": {"count": 2, "keep": 1}})
    assert chosen.tolist() == [[2, 3]] and torch.allclose(w, torch.tensor([[0.8, 0.5]], dtype=F64))
    chosen, w = plain.route(z, {"top": 2, "scale": 1.0})
    assert chosen.tolist() == [[2, 0]] and torch.allclose(w, torch.tensor([[0.4, 0.3]], dtype=F64))


# what a slip in a mechanism does to the logits of the tests' weights: planted in the plain implementation
def _one_left_out(mp):
    attend = plain.attend
    mp.setattr(plain, "attend", lambda q, k, v, s, w, one: attend(q, k, v, s, w, False))


def _window_one_longer(mp):
    attend = plain.attend
    mp.setattr(plain, "attend", lambda q, k, v, s, w, one: attend(q, k, v, s, w + 1, one))


def _half_split_rotation(mp):
    def rotate(x, rot, positions):
        d = int(rot["dims"])
        f = torch.tensor([float(rot["base"]) ** (-2.0 * i / d) for i in range(d // 2)], dtype=F64)
        a = positions.to(F64)[:, None] * f
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., :d // 2], x[..., d // 2:d]
        return torch.cat([u * c - v * s, v * c + u * s, x[..., d:]], dim=-1)
    mp.setattr(plain, "rotate", rotate)


def _no_running_maximum(mp):
    def memory(q, k, v, i, f):
        S, n = torch.zeros(*k.shape[1:], v.shape[2], dtype=F64), torch.zeros(*k.shape[1:], dtype=F64)
        out = torch.zeros(*v.shape, dtype=F64)
        for t in range(len(q)):
            S = torch.exp(f[t])[:, None, None] * S + torch.exp(i[t])[:, None, None] * k[t][:, :, None] * v[t][:, None]
            n = torch.exp(f[t])[:, None] * n + torch.exp(i[t])[:, None] * k[t]
            out[t] = torch.einsum("hdv,hd->hv", S, q[t]) / (n * q[t]).sum(-1).abs()[:, None]     # and no floor
        return out
    mp.setattr(plain, "matrix_memory", memory)


def _cap_left_out(mp):
    mp.setattr(plain, "capped", lambda z, cap: z)


def _groups_left_out(mp):
    route = plain.route
    mp.setattr(plain, "route", lambda z, r: route(z, {k: v for k, v in r.items() if k != "groups"}))


def _weights_renormalised(mp):
    route = plain.route

    def renormalised(z, r):
        chosen, w = route(z, r)
        return chosen, w / w.sum(-1, keepdim=True) * float(r["scale"])
    mp.setattr(plain, "route", renormalised)


def _relu_not_squared(mp):
    mp.setattr(plain, "squared_relu", lambda W, p, h: plain.lin(W, p + ".down", torch.relu(plain.lin(W, p + ".up", h))))


def _keys_one_token_late(mp):
    keys = plain.keys_and_values
    mp.setattr(plain, "keys_and_values", lambda *a: tuple(t.roll(1, dims=0) for t in keys(*a)))


@pytest.mark.parametrize("slip,name", [(_one_left_out, "A"), (_window_one_longer, "A"), (_half_split_rotation, "A"),
                                       (_no_running_maximum, "C"), (_cap_left_out, "B"), (_groups_left_out, "A"),
                                       (_weights_renormalised, "A"), (_relu_not_squared, "A"), (_keys_one_token_late, "A")],
                         ids=lambda f: f.__name__[1:] if callable(f) else f)
def test_a_slip_in_a_mechanism_shows_in_the_logits(slip, name, monkeypatch):
    """The engine tests' weights give every mechanism a say: a slip moves most rows by many times what the engine is
    allowed in 32-bit (2e-5).  (Norms follow the memory's read-out head by head and every sublayer's result, so that
    what only scales a result shows through their eps alone: configuration C has a large one.)"""
    import helpers
    config = CONFIGS[name]
    W = plain.random_tensors(config, 23 + ord(name))
    toks = helpers.random_tokens(61, config["vocab"], 253)
    want = plain.forward(W, config, toks)
    slip(monkeypatch)
    err = (plain.forward(W, config, toks) - want).abs().max(-1).values / want.abs().max()
    assert float((err > 4e-4).double().mean()) > 0.5, float(err.max())
