"""Python faces of the kernels of linear attention in its recurrent form and of the norm that follows a gated sum;
see ``ops/__init__.py``."""
from __future__ import annotations

from typing import Optional

import torch

from . import AP_F32, KernelError, _check, _partials, call, core, dtype_code, stream_handle

DECAY_MODES = {"head": 0, "head_token": 1, "channel": 2, "channel_token": 3, "head_ready": 4}
QK_MODES = {None: 0, "plain": 0, "rotate": 1, "unit": 2, "silu": 3}
GATE_ACTIVATIONS = {"silu": 0, "sigmoid": 1}


def _rows32(t: torch.Tensor, name: str, T: int, width: int):
    """(pointer, row stride) of a 32-bit matrix view ``[T, width]`` with contiguous rows (it may be a run of
    columns of a wider matrix)."""
    if t.dtype != torch.float32 or t.dim() != 2 or not t.is_cuda or t.stride(1) != 1 or t.shape[0] < T \
            or t.shape[1] != width:
        raise KernelError(f"linear_scan: {name} must be 32-bit [T, {width}] with contiguous rows, is "
                          f"{tuple(t.shape)} {t.dtype}")
    return t.data_ptr(), t.stride(0)


def linear_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, y: torch.Tensor, state: torch.Tensor,
                seq_start: torch.Tensor, positions: torch.Tensor, state_slots: torch.Tensor, num_seqs: int,
                heads: int, qk_heads: int, key_dim: int, value_dim: int, decay: str,
                decay_channel: Optional[torch.Tensor] = None, tau: float = 1.0,
                decay_head: Optional[torch.Tensor] = None, decay_const: Optional[torch.Tensor] = None,
                dt_bias: Optional[torch.Tensor] = None, beta: Optional[torch.Tensor] = None,
                qk: Optional[str] = None, cos_sin: Optional[torch.Tensor] = None, unit_eps: float = 0.0,
                out_scale: float = 1.0, workspace=None, write_gate: Optional[torch.Tensor] = None,
                unit_column: bool = False) -> None:
    """Linear attention as a recurrence over each sequence's rows, all 32-bit:
    ``S = diag(a_t) S + k_t u_t^T``, ``y_t = S^T q_t * out_scale`` with a state ``[key_dim, value_dim]`` per head.

    ``q``, ``k`` ``[T, qk_heads * key_dim]``, ``v`` ``[T, heads * value_dim]`` (views of columns of a wider
    32-bit matrix are taken); value head ``h`` reads query/key head ``h // (heads / qk_heads)``.
    ``decay``: ``"head"``: ``a = decay_const[h]``; ``"head_token"``: ``a = exp(-exp(decay_const[h]) *
    softplus(decay_head[t, h] + dt_bias[h]))``; ``"channel"``: ``a[d] = sigmoid(decay_channel[t, h, d])^(1/tau)``;
    ``"channel_token"``: ``a[d] = exp(-exp(decay_const[h]) * softplus(decay_channel[t, h, d] + dt_bias[h, d]))``.
    ``"head_ready"``: ``a = decay_head[t, h]`` itself.
    ``write_gate [T, heads]``: ``u = write_gate[t, h] v``.  ``unit_column``: the values have one more column that is always
    1 (``v`` still brings ``value_dim`` of them): the state is ``[key_dim, value_dim + 1]`` per head, ``y [T, heads *
    (value_dim + 1)]``.
    ``beta [T, heads]`` (raw): the delta rule, ``u = sigmoid(beta) (v - S^T k)`` on the decayed state; else
    ``u = v``.  ``qk``: ``"rotate"`` turns the first ``2 * cos_sin.shape[1]`` coordinates of every query and key
    head by ``cos_sin [T, r/2, 2]``; ``"unit"`` divides each by ``sqrt(sum x^2 + unit_eps)``; ``"silu"`` puts queries,
    keys AND values under SiLU.
    ``state [slots, heads, key_dim, value_dim]`` may be a strided view of the slots' rows; a sequence whose first
    row has position 0 starts from zero.  ``q``, ``k``, ``v``, ``decay_channel``, ``decay_head`` and ``beta`` are
    scratch: a pass before the recurrence turns them into what it reads (rotated, unit or activated vectors, decays,
    gates) in place.

    With ``workspace`` (where the buffer between its two kernels comes from) a step whose sequences bring several rows
    runs eight tokens at a time; without it, token after token."""
    T = y.shape[0]
    if decay not in DECAY_MODES or qk not in QK_MODES:
        raise KernelError(f"linear_scan: decay {decay!r} or qk {qk!r} is not known")
    if beta is not None and write_gate is not None:
        raise KernelError("linear_scan: the delta rule has a gate of its own")
    qp, ldq = _rows32(q, "q", T, qk_heads * key_dim)
    kp, ldk = _rows32(k, "k", T, qk_heads * key_dim)
    vp, ldv = _rows32(v, "v", T, heads * value_dim)
    value_dim += 1 if unit_column else 0                     # of the state and the read-out
    yp, ldy = _rows32(y, "y", T, heads * value_dim)
    dcp = dcl = dhp = dhl = bp = bl = 0
    if decay in ("channel", "channel_token"):
        dcp, dcl = _rows32(decay_channel, "decay_channel", T, heads * key_dim)
    if decay in ("head_token", "head_ready"):
        dhp, dhl = _rows32(decay_head, "decay_head", T, heads)
    if decay not in ("channel", "head_ready"):
        _check(decay_const, "decay_const", torch.float32, 1)
        if decay_const.shape[0] != heads:
            raise KernelError("linear_scan: one decay constant per head is needed")
    if dt_bias is not None:
        _check(dt_bias, "dt_bias", torch.float32, 1)
        if dt_bias.shape[0] != (heads * key_dim if decay == "channel_token" else heads):
            raise KernelError("linear_scan: dt_bias must have one entry per decay")
    if beta is not None or write_gate is not None:
        bp, bl = _rows32(beta if beta is not None else write_gate, "the write's gate", T, heads)
    rot = 0
    if QK_MODES[qk] == 1:
        _check(cos_sin, "cos_sin", torch.float32, 3)
        rot = 2 * cos_sin.shape[1]
        if cos_sin.shape[0] < T or cos_sin.shape[2] != 2 or rot > key_dim:
            raise KernelError(f"linear_scan: cos_sin {tuple(cos_sin.shape)} is not [T, r/2, 2] with r <= {key_dim}")
    if state.dtype != torch.float32 or state.dim() != 4 or tuple(state.shape[1:]) != (heads, key_dim, value_dim) \
            or state.stride(3) != 1 or state.stride(2) != value_dim or state.stride(1) != key_dim * value_dim:
        raise KernelError(f"linear_scan: the state must be 32-bit [slots, {heads}, {key_dim}, {value_dim}] with "
                          f"contiguous heads")
    for t, n in ((seq_start, "seq_start"), (positions, "positions"), (state_slots, "state_slots")):
        _check(t, n, torch.int32, 1)
    lib, scratch = core(), 0
    if workspace is not None:
        block = int(lib.ap_linear_scan_block(T, int(num_seqs), int(heads), int(key_dim), int(value_dim), DECAY_MODES[decay]))
        if block > 0:
            blocks = (T // 8 + int(num_seqs)) * int(heads)
            scratch = workspace.get("linear_scan.blocks", (blocks * block,), torch.float32).data_ptr()
    call(lib, "ap_linear_scan", qp, ldq, kp, ldk, vp, ldv, dcp, dcl, dhp, dhl,
         decay_const.data_ptr() if decay_const is not None else 0, dt_bias.data_ptr() if dt_bias is not None else 0,
         bp, bl, cos_sin.data_ptr() if rot else 0, rot, state.data_ptr(), state.stride(0), seq_start.data_ptr(),
         positions.data_ptr(), state_slots.data_ptr(), yp, ldy, T, int(num_seqs), int(heads), int(qk_heads),
         int(key_dim), int(value_dim), DECAY_MODES[decay], QK_MODES[qk], 1 if beta is not None else 0,
         1 if unit_column else 0, float(tau), float(unit_eps), float(out_scale), scratch, stream_handle())


def exp_gates(raw_i: torch.Tensor, raw_f: torch.Tensor, bias_i: Optional[torch.Tensor], bias_f: Optional[torch.Tensor],
              cap: float, state: torch.Tensor, seq_start: torch.Tensor, positions: torch.Tensor,
              state_slots: torch.Tensor, floor: torch.Tensor, num_seqs: int) -> None:
    """Exponential gates per head and token under a running maximum, all 32-bit.  With ``i = cap tanh((raw_i + bias_i) /
    cap)``, ``f = logsigmoid(cap tanh((raw_f + bias_f) / cap))`` and ``m = max(f + m, i)`` along each sequence (``state
    [slots, heads]``, may be a strided view of the slots' rows, carries ``m``; a sequence whose first row has position 0
    starts from 0): ``raw_f`` becomes the decay ``exp(f + m_before - m)``, ``raw_i`` the write's gate ``exp(i - m)``, both
    ``[T, heads]`` in place (they may be runs of columns of one wider matrix), and ``floor [T, heads]`` ``exp(-m)``."""
    _check(floor, "floor", torch.float32, 2)
    T, heads = floor.shape
    ip, ldi = _rows32(raw_i, "raw_i", T, heads)
    fp, ldf = _rows32(raw_f, "raw_f", T, heads)
    if ldi != ldf:
        raise KernelError("exp_gates: both gates must have the same row stride")
    for t, n in ((bias_i, "bias_i"), (bias_f, "bias_f")):
        if t is not None:
            _check(t, n, torch.float32, 1)
            if t.shape[0] != heads:
                raise KernelError(f"exp_gates: {n} must have one entry per head")
    if state.dtype != torch.float32 or state.dim() != 2 or state.shape[1] != heads or state.stride(1) != 1 or not state.is_cuda:
        raise KernelError(f"exp_gates: the state must be 32-bit [slots, {heads}] with contiguous rows")
    for t, n in ((seq_start, "seq_start"), (positions, "positions"), (state_slots, "state_slots")):
        _check(t, n, torch.int32, 1)
    call(core(), "ap_exp_gates", ip, fp, ldi, bias_i.data_ptr() if bias_i is not None else 0,
         bias_f.data_ptr() if bias_f is not None else 0, float(cap), state.data_ptr(), state.stride(0),
         seq_start.data_ptr(), positions.data_ptr(), state_slots.data_ptr(), floor.data_ptr(), T, int(num_seqs), heads,
         stream_handle())


def head_norm_gate(y: torch.Tensor, gate: torch.Tensor, weight: Optional[torch.Tensor], eps: float,
                   out: torch.Tensor, heads: int, value_dim: int, out_scale: float = 1.0,
                   activation: str = "silu", floor: Optional[torch.Tensor] = None, floor_eps: float = 0.0) -> None:
    """``out[t, h] = y[t, h] / sqrt(mean(y[t, h]^2) + eps) * weight * act(gate[t, h]) * out_scale`` per head of
    ``value_dim`` numbers; ``y`` and ``gate`` 32-bit ``[T, heads * value_dim]`` (may be runs of columns of a
    wider matrix), ``weight`` 32-bit ``[value_dim]`` shared by the heads, ``[heads * value_dim]`` or None; ``activation``
    ``"silu"`` or ``"sigmoid"``.  A norm over several heads together is one head of their whole width.  With ``floor
    [T, heads]`` a head of ``y`` has one more number (``y [T, heads * (value_dim + 1)]``), and the head is first divided
    by ``max(|that number|, floor) + floor_eps``."""
    if activation not in GATE_ACTIVATIONS:
        raise KernelError(f"head_norm_gate: gate activation {activation!r} is not known")
    T = out.shape[0]
    _check(out, "out", dims=2)
    hs, fptr = value_dim, 0
    if floor is not None:
        _check(floor, "floor", torch.float32, 2)
        if floor.shape[0] < T or floor.shape[1] != heads:
            raise KernelError("head_norm_gate: the floor must be [T, heads]")
        hs, fptr = value_dim + 1, floor.data_ptr()
    yp, ldy = _rows32(y, "y", T, heads * hs)
    gp, ldg = _rows32(gate, "gate", T, heads * value_dim)
    if out.shape[1] != heads * value_dim:
        raise KernelError("head_norm_gate: out must be [T, heads * value_dim]")
    own = 0
    if weight is not None:
        _check(weight, "weight", torch.float32, 1)
        if weight.shape[0] not in (value_dim, heads * value_dim):
            raise KernelError("head_norm_gate: the weight must have one entry per coordinate of a head, or of all heads")
        own = 1 if weight.shape[0] == heads * value_dim else 0
    call(core(), "ap_head_norm_gate", yp, ldy, hs, fptr, float(floor_eps), gp, ldg,
         weight.data_ptr() if weight is not None else 0, own, float(eps),
         float(out_scale), GATE_ACTIVATIONS[activation], out.data_ptr(), dtype_code(out.dtype), T, int(heads),
         int(value_dim), stream_handle())


def gated_postnorm(x: torch.Tensor, weight: torch.Tensor, groups: int, eps: float, alpha: float = 1.0,
                   delta: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None,
                   gate_bias: Optional[torch.Tensor] = None, copy: Optional[torch.Tensor] = None,
                   rows: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None) -> None:
    """The norm after a sum: ``v = alpha * x + sigmoid(gate + gate_bias) * sum(delta)``, then every one of the
    ``groups`` equal runs of ``v`` over its own ``sqrt(mean(run^2) + eps)``, times ``weight``; all 32-bit.

    Without ``rows``: ``x`` (32-bit ``[T, H]``) is overwritten with the result, and ``copy`` (optional, any type)
    receives it too.  With ``rows`` (int32 indices) or ``out`` alone: the chosen (or all) rows are normed into
    ``out`` and ``x`` stays.  ``delta``: 32-bit partial sums ``[S, T, H]`` or ``[T, H]``; ``gate``: 32-bit ``[T, H]``
    raw (may be a run of columns of a wider matrix), ``gate_bias [H]``."""
    _check(x, "x", torch.float32, 2)
    _check(weight, "weight", dims=1)
    T, H = x.shape
    if weight.shape[0] != H:
        raise KernelError("gated_postnorm: the weight must have one entry per column")
    S, dptr, dstride = 0, 0, 0
    if delta is not None:
        dptr, code, S, dstride, dT, dN = _partials(delta, "delta")
        if code != AP_F32 or dT != T or dN != H:
            raise KernelError(f"gated_postnorm: delta {tuple(delta.shape)} {delta.dtype} does not match x {tuple(x.shape)}")
    gptr = gld = 0
    if gate is not None:
        if gate.dtype != torch.float32 or gate.dim() != 2 or gate.stride(1) != 1 or gate.shape[0] < T \
                or gate.shape[1] != H or not gate.is_cuda:
            raise KernelError("gated_postnorm: the gate must be 32-bit [T, H] with contiguous rows")
        gptr, gld = gate.data_ptr(), gate.stride(0)
    if gate_bias is not None:
        _check(gate_bias, "gate_bias", torch.float32, 1)
    update = rows is None and out is None
    target = copy if update else out
    R = T
    if rows is not None:
        _check(rows, "rows", torch.int32, 1)
        R = rows.shape[0]
    if target is not None:
        _check(target, "out", dims=2)
        if target.shape[0] < R or target.shape[1] != H:
            raise KernelError("gated_postnorm: the output has too few rows or another width")
    elif not update:
        raise KernelError("gated_postnorm: chosen rows need an output")
    call(core(), "ap_gated_postnorm", x.data_ptr(), rows.data_ptr() if rows is not None else 0, R, dptr, S, dstride,
         gptr, gld, gate_bias.data_ptr() if gate_bias is not None else 0, float(alpha), weight.data_ptr(),
         dtype_code(weight.dtype), int(groups), float(eps), 1 if update else 0,
         target.data_ptr() if target is not None else 0, dtype_code(target.dtype) if target is not None else AP_F32,
         H, stream_handle())


def gated_row_add(delta: torch.Tensor, other: torch.Tensor, h: torch.Tensor, g: torch.Tensor) -> None:
    """``delta[t] += sigmoid(h[t] . g) * other[t]``: 32-bit ``delta``, ``other`` ``[T, H]``; ``h [T, H]`` the rows
    the gate is read off, ``g [H]``."""
    _check(delta, "delta", torch.float32, 2)
    _check(other, "other", torch.float32, 2)
    _check(h, "h", dims=2)
    T, H = delta.shape
    g = g.reshape(-1)
    _check(g, "g", dims=1)
    if tuple(other.shape) != (T, H) or tuple(h.shape) != (T, H) or g.shape[0] != H:
        raise KernelError("gated_row_add: shapes disagree")
    call(core(), "ap_gated_row_add", delta.data_ptr(), other.data_ptr(), h.data_ptr(), dtype_code(h.dtype),
         g.data_ptr(), dtype_code(g.dtype), T, H, stream_handle())
