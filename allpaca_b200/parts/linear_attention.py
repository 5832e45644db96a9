"""Linear attention in its recurrent form: per head a state ``S`` of ``key_dim x value_dim`` 32-bit numbers
that a request carries from step to step,

    ``S_t = diag(a_t) S_{t-1} + k_t u_t^T``,   ``o_t = S_t^T q_t``,

with what differs between its kinds as parameters:

* the decay ``a_t`` (``decay = {"kind": ...}``): ``"head"``: one fixed number per head (``values``: a list; the
  retention of a head); ``"head_token"``: ``exp(-exp(A_log[h]) * softplus(W_a h + dt_bias[h]))``, one number per
  head and token (tensors ``a``, ``A_log``, ``dt_bias``); ``"channel"``: one number per key channel and token,
  ``sigmoid(z)^(1/tau)`` with ``z = W_a2 (W_a1 h) + b`` through a narrow pair of products (tensors ``a1``, ``a2``,
  ``a2.b``; ``tau``; the pair's inner width is ``rank``); ``"channel_token"``: the same pair, but
  ``exp(-exp(A_log[h]) * softplus(W_a2 (W_a1 h) + dt_bias))`` with a number ``A_log`` per head and ``dt_bias`` per
  head and channel;
* decay ``{"kind": "exp_gates", "cap", "read_eps"}``: a matrix memory with exponential gates.  Per head and token a log
  input gate ``i = cap tanh((W_i h + b_i) / cap)`` and a log forget gate ``f = logsigmoid(cap tanh((W_f h + b_f) / cap))``
  (tensors ``i``, ``i.b``, ``f``, ``f.b``); with a running maximum ``m_t = max(f + m_{t-1}, i)`` from ``m = 0``,
  ``a_t = exp(f + m_{t-1} - m_t)`` and ``u_t = exp(i - m_t) v_t``.  A vector ``n`` per head sums the keys as the state
  sums ``k v^T``, and the read-out is divided by ``max(|n . q|, exp(-m_t)) + read_eps``.  ``n`` is the state's last column:
  the values have one more column that is always 1.  ``m`` is state too;
* ``delta_rule``: the state is corrected towards the value along the key, ``u_t = beta_t (v_t - S^T k_t)`` on
  the state already decayed, ``beta = sigmoid(W_b h)`` (tensor ``b``), and the read-out sees the correction;
  else ``u_t = v_t``;
* ``conv_taps`` ``n > 0``: Q, K and V each pass a causal convolution over the last ``n`` tokens per channel
  (tensors ``q.conv``, ``k.conv``, ``v.conv`` ``[channels, n]``, the last column on the row itself, zeros before
  the sequence's start) and SiLU; the last ``n - 1`` inputs are state too;
* ``qk``: ``"rotate"`` (with ``rope``, a ``position`` part whose ``head_dim`` is the number of rotated
  coordinates) turns queries and keys by the position; ``"unit"`` makes each a unit vector,
  ``x / sqrt(sum x^2 + unit_eps)``; ``"silu"`` puts queries, keys and values under SiLU (the convolution's own SiLU
  makes that needless where there is one); None leaves them;
* ``query_scale`` and ``key_scale`` multiply queries and keys (after rotation or unit norm);
* ``qk_heads``: value head ``h`` reads query/key head ``h // (heads / qk_heads)``;
* every head's read-out is divided by its root mean square (``norm_eps``), multiplied by a weight per coordinate
  that the heads share (``norm_weight``: tensor ``norm``) or by nothing; with ``norm_weight = "row"`` every head has
  weights of its own (``norm [heads * value_dim]``); with ``norm_over = "row"`` the heads are normed together, over the
  whole row, with a weight per coordinate of the row;
* then it is multiplied by ``act(gate)`` (``gate = {"activation", "rank"}``: ``"silu"`` or ``"sigmoid"``; the gate is
  ``W_g h`` (tensor ``g``) or, with a ``rank``, ``W_g2 (W_g1 h)`` (tensors ``g1``, ``g2``)) and by ``output_scale``, and
  projected out (tensor ``o``).

Narrow pairs of products (of the decay and of the gate) run as two products together: the first matrices stacked, the
second ones as the diagonal blocks of one matrix.

What enters the recurrence is 32-bit: the stacked projection leaves 32-bit sums; decays, gates of the write,
unit norms, the state and the read-out's norm are computed in 32-bit.  The kernels read only the step's device
tensors; a portion that starts at position 0 starts from zeros.
"""
from __future__ import annotations

import dataclasses
from typing import Dict, Mapping

import torch

from .. import ops
from .base import BuildEnv, LayerCache, Mixer, PartError, Slices, WeightSpec, build, register
from .linear import Linear


DECAY_KINDS = ("head", "head_token", "channel", "channel_token", "exp_gates")


@register("mixer", "linear_recurrence")
class LinearRecurrence(Mixer):
    """Parameters: ``hidden_size``, ``heads``, ``qk_heads`` (``heads``), ``key_dim``, ``value_dim``, ``decay``,
    ``delta_rule`` (False), ``conv_taps`` (0), ``qk`` (None), ``rope``, ``unit_eps`` (1e-6), ``query_scale`` (1),
    ``key_scale`` (1), ``norm_eps``, ``norm_weight`` (True), ``norm_over`` (``"head"``), ``gate`` (SiLU of a full
    product), ``output_scale`` (1); tensors ``q``, ``k``, ``v``, ``o`` and those the parameters bring."""

    def __init__(self, params, env: BuildEnv):
        super().__init__(params, env)
        self.require("hidden_size", "heads", "key_dim", "value_dim", "decay", "norm_eps")
        p = params
        self.hidden = int(p["hidden_size"])
        self.heads = int(p["heads"])
        self.qk_heads = int(p.get("qk_heads") or self.heads)
        self.D, self.V = int(p["key_dim"]), int(p["value_dim"])
        if self.qk_heads <= 0 or self.heads % self.qk_heads:
            raise PartError(f"{self.heads} heads are not a multiple of {self.qk_heads} query/key heads")
        if not (0 < self.D <= 512 and self.V > 0):
            raise PartError(f"head sizes {self.D}/{self.V} are not ones the kernel takes (keys up to 512)")
        decay = dict(p["decay"])
        self.decay_kind = decay.get("kind")
        if self.decay_kind not in DECAY_KINDS:
            raise PartError(f"decay kind {self.decay_kind!r} is not known ({', '.join(DECAY_KINDS)})")
        self.exp_gates = self.decay_kind == "exp_gates"
        self.decay_values = None
        self.tau, self.rank = 1.0, 0
        if self.decay_kind == "head":
            self.decay_values = [float(v) for v in decay.get("values") or ()]
            if len(self.decay_values) != self.heads:
                raise PartError(f"{len(self.decay_values)} fixed decays for {self.heads} heads")
        elif self.decay_kind in ("channel", "channel_token"):
            self.tau, self.rank = float(decay.get("tau", 1.0)), int(decay.get("rank") or 0)
            if not self.tau > 0 or self.rank <= 0:
                raise PartError("a decay per channel needs a positive tau and the rank of its pair of products")
        elif self.exp_gates:
            self.cap, self.read_eps = float(decay.get("cap") or 0.0), float(decay.get("read_eps", 0.0))
            if not self.cap > 0:
                raise PartError("exponential gates need a positive cap")
        gate = dict(p.get("gate") or {})
        self.gate_act, self.gate_rank = gate.get("activation", "silu"), int(gate.get("rank") or 0)
        if self.gate_act not in ops.recurrent.GATE_ACTIVATIONS:
            raise PartError(f"gate activation {self.gate_act!r} is not known "
                            f"({', '.join(ops.recurrent.GATE_ACTIVATIONS)})")
        self.norm_over = p.get("norm_over", "head")
        if self.norm_over not in ("head", "row"):
            raise PartError(f"norm_over {self.norm_over!r} is not known (head, row)")
        self.delta_rule = bool(p.get("delta_rule", False))
        self.taps = int(p.get("conv_taps") or 0)
        self.qk = p.get("qk")
        if self.qk not in ops.recurrent.QK_MODES:
            raise PartError(f"qk {self.qk!r} is not known (rotate, unit, silu, None)")
        if self.exp_gates and (self.delta_rule or self.qk == "silu" or p.get("norm_over", "head") != "head"):
            raise PartError("exponential gates go with plain values, no delta rule and a norm per head")
        if self.qk == "silu" and self.taps > 0:
            raise PartError("a convolution activates queries, keys and values itself: qk \"silu\" is for none")
        self.position = None
        if self.qk == "rotate":
            self.require("rope")
            self.position = build("position", p["rope"], env)
            if self.position.head_dim > self.D or self.position.pairing != 0:
                raise PartError(f"a rotation of {self.position.head_dim} coordinates in half-split pairs does not "
                                f"fit heads of {self.D}")
        self.unit_eps = float(p.get("unit_eps", 1e-6))
        # S is linear in k and o in q: both scales meet in one factor on the read-out
        self.read_scale = float(p.get("query_scale", 1.0)) * float(p.get("key_scale", 1.0))
        if self.delta_rule and float(p.get("key_scale", 1.0)) != 1.0:
            raise PartError("the delta rule is not linear in the key: key_scale must be 1")
        self.norm_eps = float(p["norm_eps"])
        self.norm_weight = bool(p.get("norm_weight", True))
        self.norm_size = self.heads * self.V if "row" in (self.norm_over, p.get("norm_weight")) else self.V
        self.output_scale = float(p.get("output_scale", 1.0))
        self.qk_size, self.v_size = self.qk_heads * self.D, self.heads * self.V
        # columns of the stacked projection: q | k | v | g (unless a narrow pair forms it) | beta | decay per head, or
        # the two exponential gates
        self.cols = {"q": 0, "k": self.qk_size, "v": 2 * self.qk_size}
        total = 2 * self.qk_size + self.v_size
        if not self.gate_rank:
            self.cols["g"] = total
            total += self.v_size
        if self.delta_rule:
            self.cols["b"] = total
            total += self.heads
        if self.decay_kind == "head_token":
            self.cols["a"] = total
            total += self.heads
        if self.exp_gates:
            self.cols["i"], self.cols["f"] = total, total + self.heads
            total += 2 * self.heads
        self.in_proj = Linear(env, total, self.hidden)
        self.out_proj = Linear(env, self.hidden, self.v_size)
        # narrow pairs: (first matrix, second matrix, inner width, outputs)
        self.pairs = []
        if self.rank:
            self.pairs.append(("a1", "a2", self.rank, self.heads * self.D))
        if self.gate_rank:
            self.pairs.append(("g1", "g2", self.gate_rank, self.v_size))
        self.narrow = self.wide = None
        if self.pairs:
            inner = sum(r for _, _, r, _ in self.pairs)
            if env.dtype == torch.bfloat16:
                inner = -(-inner // 8) * 8           # rows of whole 16-byte runs, as the tensor-core products take them
            self.narrow = Linear(env, inner, self.hidden)
            self.wide = Linear(env, sum(n for _, _, _, n in self.pairs), inner)
        self.VS = self.V + (1 if self.exp_gates else 0)          # columns of a head's state
        self.matrix_floats = self.heads * self.D * self.VS
        self.state_floats = self.matrix_floats + (self.heads if self.exp_gates else 0)
        self.conv_channels = 2 * self.qk_size + self.v_size
        self.conv_floats = max(self.taps - 1, 0) * self.conv_channels
        self.norm_w = self.decay_const = self.dt_bias = self.conv_w = self.i_bias = self.f_bias = None

    def parts(self):
        yield self
        if self.position is not None:
            yield from self.position.parts()

    def weights(self) -> Dict[str, WeightSpec]:
        H = self.hidden
        w = {"q": WeightSpec((self.qk_size, H)), "k": WeightSpec((self.qk_size, H)),
             "v": WeightSpec((self.v_size, H)), "o": WeightSpec((H, self.v_size))}
        if not self.gate_rank:
            w["g"] = WeightSpec((self.v_size, H))
        for first, second, r, n in self.pairs:
            w.update({first: WeightSpec((r, H)), second: WeightSpec((n, r))})
        if self.norm_weight:
            w["norm"] = WeightSpec((self.norm_size,), "norm")
        if self.delta_rule:
            w["b"] = WeightSpec((self.heads, H))
        if self.decay_kind == "head_token":
            w.update({"a": WeightSpec((self.heads, H)), "A_log": WeightSpec((self.heads,), "bias"),
                      "dt_bias": WeightSpec((self.heads,), "bias")})
        if self.exp_gates:
            for n in ("i", "f"):
                w.update({n: WeightSpec((self.heads, H)), n + ".b": WeightSpec((self.heads,), "bias")})
        if self.decay_kind == "channel":
            w["a2.b"] = WeightSpec((self.heads * self.D,), "bias")
        if self.decay_kind == "channel_token":
            w.update({"A_log": WeightSpec((self.heads,), "bias"), "dt_bias": WeightSpec((self.heads * self.D,), "bias")})
        if self.taps > 0:
            w.update({"q.conv": WeightSpec((self.qk_size, self.taps), "bias"),
                      "k.conv": WeightSpec((self.qk_size, self.taps), "bias"),
                      "v.conv": WeightSpec((self.v_size, self.taps), "bias")})
        return w

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        stacked = [tensors["q"], tensors["k"], tensors["v"]]
        if not self.gate_rank:
            stacked.append(tensors["g"])
        if self.delta_rule:
            stacked.append(tensors["b"])
        if self.decay_kind == "head_token":
            stacked.append(tensors["a"])
        if self.exp_gates:
            stacked += [tensors["i"], tensors["f"]]
            self.i_bias, self.f_bias = (tensors[n].float().contiguous() for n in ("i.b", "f.b"))
        if self.decay_kind in ("head_token", "channel_token"):
            self.decay_const = tensors["A_log"].float().contiguous()
            self.dt_bias = tensors["dt_bias"].float().contiguous()
        self.in_proj.load(torch.cat(stacked, dim=0))
        self.out_proj.load(tensors["o"])
        if self.decay_kind == "head":
            self.decay_const = torch.tensor(self.decay_values, dtype=torch.float64).to(torch.float32).to(self.env.device)
        if self.pairs:
            self._load_pairs(tensors)
        # what enters the recurrence is 32-bit whatever the engine's type
        self.norm_w = tensors["norm"].float().contiguous() if self.norm_weight else None
        if self.taps > 0:
            self.conv_w = torch.cat([tensors["q.conv"], tensors["k.conv"], tensors["v.conv"]], dim=0).float().contiguous()

    def _load_pairs(self, tensors: Mapping[str, torch.Tensor]) -> None:
        like = tensors[self.pairs[0][0]]
        first, second = (like.new_zeros(m.out_features, m.in_features) for m in (self.narrow, self.wide))
        r0 = n0 = 0
        for a, b, r, n in self.pairs:
            first[r0:r0 + r] = tensors[a]
            second[n0:n0 + n, r0:r0 + r] = tensors[b]
            r0, n0 = r0 + r, n0 + n
        bias = None
        if self.decay_kind == "channel":
            bias = like.new_zeros(self.wide.out_features)
            bias[:self.heads * self.D] = tensors["a2.b"]
        self.narrow.load(first)
        self.wide.load(second, bias)

    def state_bytes(self) -> int:
        return 4 * (self.state_floats + self.conv_floats)

    def forward(self, h: torch.Tensor, step, cache: LayerCache, into=None) -> torch.Tensor:
        """``into`` (optional, 32-bit ``[T, hidden]``): where the output projection leaves its sums, for a mixer
        that runs beside another one."""
        T, S = h.shape[0], step.num_seqs
        ws = self.env.workspace
        if cache.state is None:
            raise PartError("a recurrent mixer needs a state slot per request")
        proj = self.in_proj.forward(h, "linrec.proj", "float32")
        rows = cache.state.view(torch.float32)
        state = rows[:, :self.matrix_floats].unflatten(1, (self.heads, self.D, self.VS))
        c = self.cols
        if self.taps > 0:
            conv_state = rows[:, self.state_floats:self.state_floats + self.conv_floats] \
                .unflatten(1, (self.taps - 1, self.conv_channels)) if self.taps > 1 else None
            qkv = ws.get("linrec.conv", (T, self.conv_channels), torch.float32)
            ops.causal_conv(proj, 0, self.conv_w, None, conv_state, step.seq_start, step.positions, step.state_slots,
                            qkv, S)
        else:
            qkv = proj
        q, k = qkv[:, c["q"]:c["q"] + self.qk_size], qkv[:, c["k"]:c["k"] + self.qk_size]
        v = qkv[:, c["v"]:c["v"] + self.v_size]
        decay_channel = None
        gate = proj[:, c["g"]:c["g"] + self.v_size] if "g" in c else None
        if self.pairs:
            wide = self.wide.forward(self.narrow.forward(h, "linrec.narrow", "either"), "linrec.wide", "float32")
            at = self.heads * self.D if self.rank else 0
            if self.rank:
                decay_channel = wide[:, :at]
            if self.gate_rank:
                gate = wide[:, at:]
        decay, decay_head, write_gate, floor = self.decay_kind, None, None, None
        if "a" in c:
            decay_head = proj[:, c["a"]:c["a"] + self.heads]
        if self.exp_gates:
            decay, decay_head = "head_ready", proj[:, c["f"]:c["f"] + self.heads]
            write_gate = proj[:, c["i"]:c["i"] + self.heads]
            floor = ws.get("linrec.floor", (T, self.heads), torch.float32)
            ops.exp_gates(write_gate, decay_head, self.i_bias, self.f_bias, self.cap,
                          rows[:, self.matrix_floats:self.state_floats], step.seq_start, step.positions,
                          step.state_slots, floor, S)
        y = ws.get("linrec.y", (T, self.heads * self.VS), torch.float32)
        ops.linear_scan(q, k, v, y, state, step.seq_start, step.positions, step.state_slots, S, self.heads,
                        self.qk_heads, self.D, self.V, decay, decay_channel=decay_channel, tau=self.tau,
                        decay_head=decay_head, write_gate=write_gate, unit_column=self.exp_gates,
                        decay_const=self.decay_const, dt_bias=self.dt_bias,
                        beta=proj[:, c["b"]:c["b"] + self.heads] if self.delta_rule else None, qk=self.qk,
                        cos_sin=self.position.rotation_for(step)[0] if self.position is not None else None,
                        unit_eps=self.unit_eps, out_scale=self.read_scale, workspace=ws)
        gated = ws.get("linrec.gated", (T, self.v_size), self.env.dtype)
        heads, V = (1, self.v_size) if self.norm_over == "row" else (self.heads, self.V)
        ops.head_norm_gate(y, gate, self.norm_w, self.norm_eps, gated, heads, V, out_scale=self.output_scale,
                           activation=self.gate_act, floor=floor, floor_eps=self.read_eps if self.exp_gates else 0.0)
        return self.out_proj.forward(gated, "linrec.o", "delta", into=into)


@register("mixer", "mixer_pair")
class MixerPair(Mixer):
    """Two mixers side by side on the same input: ``left_scale * left(h) + right_scale * right(h)``.

    Parameters: ``left``, ``right`` (:class:`PartSpec` of mixers that take ``output_scale`` as a parameter and
    ``into=`` in ``forward``), ``left_scale`` (1), ``right_scale`` (1).  Tensors: the sides' own under ``left.`` and
    ``right.``.  At most one side may keep pages; both may keep fixed-size state (the left one's first in the
    request's slot).  Each side scales its own result where that is free and leaves the sums of its output
    projection in one slice of ``[2, T, hidden]``, which whoever adds into the residual sums up.

    ``output_norm_eps`` (None: no norm): each side's result (with its projection's bias) is divided by its own root
    mean square over the model's width and multiplied by a plain weight (tensors ``left.out``, ``right.out``) before
    the sum.  :meth:`forward_slices` leaves that to the kernel that adds the result to the residual."""

    def __init__(self, params, env: BuildEnv):
        super().__init__(params, env)
        self.require("left", "right")
        self.sides = []
        eps = params.get("output_norm_eps")
        self.norm_eps = float(eps) if eps is not None else None
        self.scales = [float(params.get(name + "_scale", 1.0)) for name in ("left", "right")]
        for name, scale in zip(("left", "right"), self.scales):
            spec = params[name]
            # a norm behind a side takes a scale of its input out again: the scale goes behind the norm
            scaled = dict(spec.params, output_scale=scale if self.norm_eps is None else 1.0)
            self.sides.append((name + ".", build("mixer", type(spec)(spec.name, scaled), env)))
        self.out_weight = self.out_bias = None
        self._ones = None
        if sum(1 for _, m in self.sides if m.cache_need() is not None) > 1:
            raise PartError("only one of two mixers side by side may keep pages")
        self.hidden = int(params.get("hidden_size") or self.sides[0][1].hidden)

    def parts(self):
        yield self
        for _, m in self.sides:
            yield from m.parts()

    def weights(self) -> Dict[str, WeightSpec]:
        w = {prefix + n: ws for prefix, m in self.sides for n, ws in m.weights().items()}
        if self.norm_eps is not None:
            w.update({prefix + "out": WeightSpec((self.hidden,), "norm") for prefix, _ in self.sides})
        return w

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        for prefix, m in self.sides:
            names = set(m.weights())
            m.load({n[len(prefix):]: t for n, t in tensors.items() if n.startswith(prefix) and n[len(prefix):] in names})
        if self.norm_eps is not None:
            self.out_weight = torch.stack([tensors[prefix + "out"].float() * scale
                                           for (prefix, _), scale in zip(self.sides, self.scales)]).contiguous()
        self._ones = torch.ones(self.hidden, dtype=torch.float32, device=self.env.device)
        biases = [getattr(m, "output_bias", None) for _, m in self.sides]
        if any(b is not None for b in biases):
            self.out_bias = torch.stack([b if b is not None else torch.zeros(self.hidden, device=self.env.device)
                                         for b in biases]).contiguous()

    def cache_need(self):
        for _, m in self.sides:
            if m.cache_need() is not None:
                return m.cache_need()
        return None

    def state_bytes(self) -> int:
        return sum(m.state_bytes() for _, m in self.sides)

    def forward(self, h: torch.Tensor, step, cache: LayerCache) -> torch.Tensor:
        y = self.forward_slices(h, step, cache)
        if y.bias is None and y.weight is None:
            return y.sums
        # a block that takes plain sums: the slices finished by the kernel that applies them to one stream
        T, ws = h.shape[0], self.env.workspace
        done = ws.get("pair.done", (T, 1, self.hidden), torch.float32)
        ops.stream_norm(done, self._ones[:1], self._ones, 1.0, ws.get("pair.unused", (T, self.hidden), torch.float32),
                        delta=y.sums, out_w=self._ones[:1], slice_bias=y.bias, slice_weight=y.weight, slice_eps=y.eps)
        return done.view(1, T, self.hidden)

    def forward_slices(self, h: torch.Tensor, step, cache: LayerCache) -> Slices:
        T = h.shape[0]
        delta = self.env.workspace.get("pair.delta", (2, T, self.hidden), torch.float32)
        at = 0
        for i, (_, m) in enumerate(self.sides):
            own = m.state_bytes()
            side = cache
            if cache.state is not None:
                side = dataclasses.replace(cache, state=cache.state[:, at:at + own] if own else None)
            at += own
            if getattr(m, "output_bias", None) is not None:
                m.forward(h, step, side, into=delta[i], add_bias=False)
            else:
                m.forward(h, step, side, into=delta[i])
        return Slices(delta, self.out_bias, self.out_weight, self.norm_eps or 0.0)
