"""The Boketar decoder without a GPU: configuration, tensor names and shapes against the plain list, what each layer asks
of the cache and of the state slots, refused configurations, the sizes that the tensors' shapes give, and each
mechanism of the plain implementation by hand."""
import copy
import math

import pytest
import torch

import plain_boketar as plain
from boketar_configs import CONFIGS

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
    # layer 0: 3 key/value heads of 24 + 40 behind a window of 21; layer 2: one head of 32 + 16 behind 50
    assert [(g.need.outer, g.need.inner, g.need.window, g.runs) for g in plan] == \
        [((3,), (64,), 21, [0]), ((1,), (48,), 50, [2])]
    assert model.state_bytes() == [
        4 * (2 * (6 * 24 + 3 * 24 + 3 * 40) + 3 * 16 * 8),           # two inputs of each channel; lightning 3 x 16 x 8
        4 * (3 * 16 * 24 + 3 * (16 + 16 + 72)),                      # the delta rule's state and three inputs
        4 * ((2 * 32 + 32 + 16) + 5 * 8 * 12),
        4 * (2 * 32 * 8 + (64 + 64 + 16))]
    assert not model.host_control()
    assert model.spec.streams == 3 and cfg.embedding_scale == 3.0
    _, model = build(CONFIGS["B"])
    assert model.state_bytes()[:2] == [4 * 4 * 40 * 16, 4 * 64 * 32]  # convolutions of one tap keep no inputs


def test_refused_configurations():
    from allpaca_b200.config import BoketarConfig, ConfigError
    base = CONFIGS["A"]

    def broken(change):
        c = copy.deepcopy(base)
        change(c)
        with pytest.raises(ConfigError):
            BoketarConfig.from_dict(c)
    broken(lambda c: c["layers"][0].update(type="delta"))
    broken(lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4))               # 6 heads on 4
    broken(lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7))             # odd
    broken(lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=26))            # more than the head has
    broken(lambda c: c["layers"][0]["mixer"]["left"].pop("conv"))
    broken(lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0))
    broken(lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.9, 0.9]))         # three heads
    broken(lambda c: c["layers"][1]["mixer"].pop("decay_rank"))                         # and no tensors to read it off
    broken(lambda c: c["layers"][1]["mixer"].update(conv=0))
    broken(lambda c: c["layers"][1]["mlp"].update(kind="moe"))
    broken(lambda c: c.update(streams=0))
    broken(lambda c: c["norm"].update(eps=0.0))
    broken(lambda c: c.pop("width"))
    broken(lambda c: c.update(layers=[]))


def test_the_narrow_widths_come_from_the_tensors(tmp_path):
    """config.json need not name the inner widths of the narrow pairs of products: the checkpoint's shapes do."""
    from allpaca_b200.models import load_config
    from allpaca_b200.weights import write_model_folder
    config = copy.deepcopy(CONFIGS["A"])
    tensors = {k: v.to(torch.bfloat16) for k, v in plain.random_tensors(config, 3).items()}
    for i in (1, 3):
        del config["layers"][i]["mixer"]["decay_rank"], config["layers"][i]["mixer"]["gate_rank"]
    write_model_folder(str(tmp_path), config, tensors)
    _, cfg = load_config(str(tmp_path))
    assert [(cfg.layers[i].mixer.decay_rank, cfg.layers[i].mixer.gate_rank) for i in (1, 3)] == [(6, 10), (3, 1)]


def test_narrow_pairs_share_two_products():
    """The pairs' second matrices are the diagonal blocks of one: in bfloat16 the inner width is filled up to whole
    16-byte runs with zeros."""
    config = CONFIGS["A"]
    for dtype, inner in ((torch.float32, 16), (torch.bfloat16, 16)):
        _, model = build(config, dtype)
        tensors = {k: v.to(dtype) for k, v in plain.random_tensors(config, 3).items()}
        model.load_weights(tensors)
        m = model.blocks[1].mixer
        assert m.narrow.weight.shape == (inner, 64) and m.wide.weight.shape == (3 * 16 + 3 * 24, inner)
        x = torch.randn(5, 64, dtype=F64)
        both = (x @ m.narrow.weight.double().T) @ m.wide.weight.double().T
        W = {k: v.double() for k, v in tensors.items()}
        assert torch.allclose(both[:, :48], (x @ W["l1.mix.a1"].T) @ W["l1.mix.a2"].T)
        assert torch.allclose(both[:, 48:], (x @ W["l1.mix.g1"].T) @ W["l1.mix.g2"].T)
    _, model = build(config, torch.bfloat16)
    assert model.blocks[3].mixer.narrow.out_features == 8          # 3 + 1, filled up


def test_mechanisms_by_hand():
    # the streams: u = sum in x; x_t <- sum_s mix[s, t] x_s + out[t] y (the matrix is [from, to])
    xs = torch.tensor([[[1.0], [10.0]]], dtype=F64)
    assert float(plain.gather_streams(xs, torch.tensor([2.0, 0.5], dtype=F64))) == 7.0
    new = plain.scatter_streams(xs, torch.tensor([[100.0]], dtype=F64), torch.tensor([1.0, 3.0], dtype=F64),
                                torch.tensor([[1.0, 2.0], [0.0, 5.0]], dtype=F64))
    assert new.flatten().tolist() == [1.0 + 100.0, 2.0 + 50.0 + 300.0]
    # a norm weight of zero leaves the normed row
    x = torch.tensor([[3.0, 4.0]], dtype=F64)
    assert torch.allclose(plain.norm(x, torch.tensor([0.0, 1.0], dtype=F64), 0.0),
                          torch.tensor([[3.0, 8.0]], dtype=F64) / math.sqrt(12.5))
    # neighbouring coordinates turn together, the rest pass
    r = plain.rotate(torch.tensor([[[1.0, 0.0, 1.0, 0.0, 7.0]]], dtype=F64), {"base": 100.0, "dims": 4}, torch.tensor([2]))
    a = 2 * 100.0 ** -0.5
    assert torch.allclose(r[0, 0], torch.tensor([math.cos(2.0), math.sin(2.0), math.cos(a), math.sin(a), 7.0], dtype=F64))
    # the convolution's last tap is the row's own; nothing before the start; no activation
    c = plain.short_conv(torch.tensor([[1.0], [2.0], [3.0]], dtype=F64), torch.tensor([[0.5, 0.0, -2.0]], dtype=F64))
    assert c[:, 0].tolist() == [-2.0, -4.0, -5.5]
    # a window of 2 and a sink of log 2: the weights of equal scores are 1 / (n + 2)
    v = torch.tensor([[[1.0]], [[2.0]], [[4.0]]], dtype=F64)
    out = plain.attend(torch.ones(3, 1, 1, dtype=F64), torch.zeros(3, 1, 1, dtype=F64), v, 1.0, 2,
                       torch.tensor([math.log(2.0)], dtype=F64))
    assert torch.allclose(out[:, 0, 0], torch.tensor([1 / 3, 3 / 4, 6 / 4], dtype=F64))
    # the delta rule: a full gate writes the value itself at its key, whatever was there; a channel forgets on its own
    k = torch.eye(2, dtype=F64)[:, None, :]
    q = torch.tensor([[[1.0, 1.0]], [[1.0, 1.0]]], dtype=F64)
    decay = torch.tensor([[[1.0, 1.0]], [[0.25, 1.0]]], dtype=F64)
    o = plain.delta_recurrence(q, k, torch.tensor([[[8.0]], [[5.0]]], dtype=F64), decay, torch.ones(2, 1, dtype=F64))
    assert o.flatten().tolist() == [8.0, 2.0 + 5.0]


# what a slip in a mechanism does to the logits of the tests' weights: planted in the plain implementation
def _sink_left_out(mp):
    attend = plain.attend
    mp.setattr(plain, "attend", lambda q, k, v, s, w, sink: attend(q, k, v, s, w, None))


def _window_one_longer(mp):
    attend = plain.attend
    mp.setattr(plain, "attend", lambda q, k, v, s, w, sink: attend(q, k, v, s, w + 1, sink))


def _half_split_rotation(mp):
    def rotate(x, rot, positions):
        d = int(rot["dims"])
        f = torch.tensor([float(rot["base"]) ** (-2.0 * i / d) for i in range(d // 2)], dtype=F64)
        a = positions.to(F64)[:, None] * f
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., :d // 2], x[..., d // 2:d]
        return torch.cat([u * c - v * s, v * c + u * s, x[..., d:]], dim=-1)
    mp.setattr(plain, "rotate", rotate)


def _mix_transposed(mp):
    scatter = plain.scatter_streams
    mp.setattr(plain, "scatter_streams", lambda xs, y, o, m: scatter(xs, y, o, m.T))


def _norm_weight_plain(mp):
    norm = plain.norm
    mp.setattr(plain, "norm", lambda x, w, eps: norm(x, w - 1.0, eps))


def _sides_summed_whole(mp):
    halves = plain.normed_halves
    mp.setattr(plain, "normed_halves", lambda a, b, wa, wb, eps: 0.5 * (a * wa + b * wb))


def _decay_after_the_write(mp):
    rec = plain.delta_recurrence
    mp.setattr(plain, "delta_recurrence", lambda q, k, v, d, b: rec(q, k, v, torch.cat([torch.ones_like(d[:1]), d[:-1]]), b))


def _one_decay_for_all_channels(mp):
    decay = plain.channel_decay
    mp.setattr(plain, "channel_decay", lambda *a: decay(*a).mean(-1, keepdim=True).expand(decay(*a).shape))


def _convolution_skips_a_token(mp):
    conv = plain.short_conv
    mp.setattr(plain, "short_conv", lambda x, w: conv(x, torch.cat([w[:, 1:2], w[:, :1], w[:, 2:]], dim=1)))


@pytest.mark.parametrize("slip", [_sink_left_out, _window_one_longer, _half_split_rotation, _mix_transposed,
                                  _norm_weight_plain, _sides_summed_whole, _decay_after_the_write,
                                  _one_decay_for_all_channels, _convolution_skips_a_token], ids=lambda f: f.__name__[1:])
def test_a_slip_in_a_mechanism_shows_in_the_logits(slip, monkeypatch):
    """The engine tests' weights give every mechanism a say: a slip moves more rows beyond the tolerances the engine is
    held to (2e-5 in 32-bit; 3 % in bfloat16 but for one row in fifty) than those allow."""
    import helpers
    config = CONFIGS["A"]
    W = plain.random_tensors(config, 23 + ord("A"))
    toks = helpers.random_tokens(61, config["vocab"], 253)
    want = plain.forward(W, config, toks)
    slip(monkeypatch)
    err = ((plain.forward(W, config, toks) - want) ** 2).mean(-1).sqrt() / (want ** 2).mean().sqrt()
    assert float((err > 0.04).double().mean()) > 0.1, float(err.max())
