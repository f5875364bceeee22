"""Kernels of mixers that keep a state of fixed size per request: the linear scan (plain or delta
rule, constant or per-row decay), the short convolution's bookkeeping, and the gated group norm of
the read-out.  The state and everything that enters the recurrence are float32."""

from __future__ import annotations

import torch

from ..errors import KernelError
from .native import call, ptr, require, stream_ptr, tag


def linear_scan(
    q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, *, heads: int, qk_heads: int, dim: int, vdim: int,
    state: torch.Tensor, q_start: torch.Tensor, slots: torch.Tensor, gate: torch.Tensor | None = None,
    decay: torch.Tensor | None = None, beta: torch.Tensor | None = None, silu: bool = False, q_scale: float = 1.0,
    fixed_order: bool = False, row_decay: torch.Tensor | None = None,
) -> torch.Tensor:
    """Per request (entry ``e`` owns rows ``q_start[e] .. q_start[e+1]-1`` and the state row ``slots[e]``) and head,
    token after token: ``S <- D S + k u^T``, ``o = S^T q`` with ``D`` the head's constant ``decay`` or the row's
    ``gate`` factors (one per key channel) or, with ``beta``, the row's one factor per head ``row_decay`` (``[N, heads]``), and ``u = v``
    or, with ``beta``, ``beta (v - (D S)^T k)``.  ``q`` and
    ``k`` are ``[N, qk_heads * dim]`` column blocks (a row stride of their own is fine), ``v`` ``[N, heads * vdim]``;
    head ``h`` reads q/k head ``h // (heads / qk_heads)``.  ``silu`` applies SiLU to q, k and v as they are read;
    q is multiplied by ``q_scale`` then.  ``v`` may be bfloat16 beside float32 ``q`` and ``k`` (constant decay, no ``beta``).
    ``state`` is ``[slots, heads, dim, vdim]`` float32 and is updated in place.  ``fixed_order``: every sum is formed in
    an order that does not depend on the shape of the batch (the kernel otherwise spreads a column over more lanes when few
    requests bring long portions), so a token's bits do not depend on the cut.  Returns float32 ``[N, heads * vdim]``."""

    n = q.shape[0]
    for t, name, width in ((q, "q", qk_heads * dim), (k, "k", qk_heads * dim), (v, "v", heads * vdim)):
        if t.device.type != "cuda" or t.dim() != 2 or t.shape != (n, width) or t.stride(1) != 1 or (name == "k" and t.dtype != q.dtype):
            raise KernelError(f"{name} must be CUDA rows [{n}, {width}] with unit column stride, q and k of one type")
    if v.dtype != q.dtype and (beta is not None or decay is None or q.dtype != torch.float32):
        raise KernelError("linear_scan takes v in another type than q and k with a constant decay and float32 q and k only")
    require(state, "state", dtype=torch.float32, dims=4)
    if tuple(state.shape[1:]) != (heads, dim, vdim):
        raise KernelError(f"state has shape {tuple(state.shape)}, expected [slots, {heads}, {dim}, {vdim}]")
    require(q_start, "q_start", dtype=torch.int32, dims=1)
    entries = q_start.shape[0] - 1
    require(slots, "slots", dtype=torch.int32, shape=(entries,))
    if sum(t is not None for t in (gate, decay, row_decay)) != 1:
        raise KernelError("linear_scan takes one of: gate factors per row and channel, one decay per row and head, one decay per head")
    if row_decay is not None:
        require(row_decay, "row_decay", dtype=torch.float32, shape=(n, heads))
        if beta is None:
            raise KernelError("linear_scan takes one decay per row and head with the delta rule only (linear_scan_row_gates otherwise)")
    elif gate is not None:
        require(gate, "gate", dtype=torch.float32, shape=(n, heads * dim))
    else:
        require(decay, "decay", dtype=torch.float32, shape=(heads,))
    if beta is not None:
        require(beta, "beta", dtype=torch.float32, shape=(n, heads))
    out = torch.empty((n, heads * vdim), dtype=torch.float32, device=q.device)
    call("b200_linear_scan", ptr(q), ptr(k), ptr(v), q.stride(0), k.stride(0), v.stride(0), ptr(gate), heads * dim, ptr(decay),
         ptr(row_decay), ptr(beta), heads, ptr(state), ptr(out), heads * vdim, ptr(q_start), ptr(slots), entries, n, heads, qk_heads, dim, vdim,
         1 if silu else 0, float(q_scale), 1 if fixed_order else 0, tag(q.dtype), tag(v.dtype), stream_ptr())
    return out


def linear_scan_row_gates(
    q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, *, heads: int, dim: int, vdim: int, decay: torch.Tensor, gain: torch.Tensor,
    state: torch.Tensor, norm_state: torch.Tensor, q_start: torch.Tensor, slots: torch.Tensor, q_scale: float = 1.0,
    fixed_order: bool = False,
) -> tuple[torch.Tensor, torch.Tensor]:
    """``linear_scan`` with one decay and one input gain per row and head, and a normaliser: ``S <- decay S + gain k v^T``,
    ``n <- decay n + gain k``; returns ``S^T q`` float32 ``[N, heads * vdim]`` and ``n . q`` float32 ``[N, heads]`` (q times
    ``q_scale`` as it is read).  ``state`` ``[slots, heads, dim, vdim]`` and ``norm_state`` ``[slots, heads, dim]`` float32 are
    updated in place; ``decay`` and ``gain`` are float32 ``[N, heads]``.  ``fixed_order`` as for ``linear_scan``."""

    n = q.shape[0]
    for t, name, width in ((q, "q", heads * dim), (k, "k", heads * dim), (v, "v", heads * vdim)):
        if t.device.type != "cuda" or t.dim() != 2 or t.shape != (n, width) or t.stride(1) != 1 or t.dtype != q.dtype:
            raise KernelError(f"{name} must be CUDA rows [{n}, {width}] of one type with unit column stride")
    require(state, "state", dtype=torch.float32, dims=4)
    require(norm_state, "norm_state", dtype=torch.float32, dims=3)
    if tuple(state.shape[1:]) != (heads, dim, vdim) or tuple(norm_state.shape[1:]) != (heads, dim) or norm_state.shape[0] != state.shape[0]:
        raise KernelError(f"states have shapes {tuple(state.shape)} and {tuple(norm_state.shape)}, expected [slots, {heads}, {dim}, {vdim}] "
                          f"and [slots, {heads}, {dim}]")
    require(decay, "decay", dtype=torch.float32, shape=(n, heads))
    require(gain, "gain", dtype=torch.float32, shape=(n, heads))
    require(q_start, "q_start", dtype=torch.int32, dims=1)
    entries = q_start.shape[0] - 1
    require(slots, "slots", dtype=torch.int32, shape=(entries,))
    out = torch.empty((n, heads * vdim), dtype=torch.float32, device=q.device)
    norm_out = torch.empty((n, heads), dtype=torch.float32, device=q.device)
    call("b200_linear_scan_row_gates", ptr(q), ptr(k), ptr(v), q.stride(0), k.stride(0), v.stride(0), ptr(decay), ptr(gain), ptr(state),
         ptr(norm_state), ptr(out), ptr(norm_out), ptr(q_start), ptr(slots), entries, n, heads, dim, vdim, float(q_scale),
         1 if fixed_order else 0, tag(q.dtype), stream_ptr())
    return out, norm_out


def memory_gates(
    proj: torch.Tensor, *, heads: int, i_offset: int, f_offset: int, i_bias: torch.Tensor, f_bias: torch.Tensor, cap: float,
    m_state: torch.Tensor, q_start: torch.Tensor, slots: torch.Tensor,
) -> tuple[torch.Tensor, torch.Tensor, torch.Tensor]:
    """Exponential gates kept in range by a running maximum.  With ``i = cap tanh((zi + i_bias) / cap)`` and
    ``f = ln sigmoid(cap tanh((zf + f_bias) / cap))`` (logits: columns ``i_offset + h`` and ``f_offset + h`` of ``proj``), token after
    token: ``m_t = max(f + m_(t-1), i)`` from the slot's ``m`` (``m_state`` float32 ``[slots, heads]``, updated in place).  Returns
    float32 ``[N, heads]`` each: ``exp(f + m_(t-1) - m_t)``, ``exp(i - m_t)`` and ``exp(-m_t)``."""

    require(proj, "proj", dims=2)
    n, ld = proj.shape
    require(i_bias, "i_bias", dtype=torch.float32, shape=(heads,))
    require(f_bias, "f_bias", dtype=torch.float32, shape=(heads,))
    require(m_state, "m_state", dtype=torch.float32, dims=2)
    if m_state.shape[1] != heads or max(i_offset, f_offset) + heads > ld:
        raise KernelError("memory_gates: the logits lie outside the rows, or the state has another number of heads")
    require(q_start, "q_start", dtype=torch.int32, dims=1)
    entries = q_start.shape[0] - 1
    require(slots, "slots", dtype=torch.int32, shape=(entries,))
    decay, gain, floor = torch.empty((3, n, heads), dtype=torch.float32, device=proj.device)
    call("b200_memory_gates", ptr(proj), ld, i_offset, f_offset, ptr(i_bias), ptr(f_bias), float(cap), ptr(m_state), ptr(decay), ptr(gain),
         ptr(floor), ptr(q_start), ptr(slots), entries, heads, tag(proj.dtype), stream_ptr())
    return decay, gain, floor


def channel_decay(proj: torch.Tensor, up: torch.Tensor, bias: torch.Tensor, *, offset: int, tau: float) -> torch.Tensor:
    """Decays per key channel from a low-rank map: ``sigmoid(proj[:, offset : offset + rank] @ up + bias)^(1 / tau)``, float32
    ``[N, width]``; ``up`` is ``[rank, width]`` (the map's weight transposed) in the type of ``proj``."""

    require(proj, "proj", dims=2)
    n, ld = proj.shape
    require(up, "up", dtype=proj.dtype, dims=2)
    rank, width = up.shape
    require(bias, "bias", dtype=torch.float32, shape=(width,))
    if offset + rank > ld:
        raise KernelError("channel_decay: the low-rank columns lie outside the rows")
    alpha = torch.empty((n, width), dtype=torch.float32, device=proj.device)
    call("b200_channel_decay", ptr(proj), ld, offset, rank, ptr(up), ptr(bias), float(tau), ptr(alpha), n, width, tag(proj.dtype),
         stream_ptr())
    return alpha


def delta_prepare(
    proj: torch.Tensor, *, heads: int, qk_heads: int, dim: int, vdim: int, beta_offset: int, low_offset: int, rank: int,
    taps: torch.Tensor, conv_state: torch.Tensor, a_log: torch.Tensor, dt_bias: torch.Tensor, a_up: torch.Tensor | None,
    q_start: torch.Tensor, slots: torch.Tensor, token_entry: torch.Tensor, unit_eps: float, q_scale: float,
):
    """From one stacked projection ``[N, q | k | v | ...]``: the short convolution over time and SiLU of every q, k
    and v channel (inputs before the step come from ``conv_state`` ``[slots, taps-1, channels]``), each q and k head
    divided by ``sqrt(sum of squares + unit_eps)`` (q times ``q_scale``), ``beta = sigmoid(proj[:, beta_offset + h])``
    and the decay factors ``exp(-exp(a_log[h]) * softplus(proj[:, low_offset : low_offset + rank] @ a_up + dt_bias))``
    (``a_up`` is ``[rank, heads * dim]``: the map's weight transposed, so that neighbouring threads read neighbouring outputs).
    ``rank`` 0 (``a_up`` ``None``): one decay per head, ``exp(-exp(a_log[h]) * softplus(proj[:, low_offset + h] + dt_bias[h]))``, and ``g``
    is ``[N, heads]``.
    Returns float32 ``(q, k, v, g, beta)``."""

    require(proj, "proj", dims=2)
    n, ld = proj.shape
    channels = 2 * qk_heads * dim + heads * vdim
    require(taps, "taps", dtype=torch.float32, dims=2)
    ntaps = taps.shape[1]
    if taps.shape[0] != channels:
        raise KernelError(f"taps has {taps.shape[0]} channels, expected {channels}")
    require(conv_state, "conv_state", dtype=torch.float32, dims=3)
    if tuple(conv_state.shape[1:]) != (ntaps - 1, channels):
        raise KernelError(f"conv_state has shape {tuple(conv_state.shape)}, expected [slots, {ntaps - 1}, {channels}]")
    require(a_log, "a_log", dtype=torch.float32, shape=(heads,))
    decays = heads * dim if rank else heads
    require(dt_bias, "dt_bias", dtype=torch.float32, shape=(decays,))
    if rank:
        require(a_up, "a_up", dtype=proj.dtype, shape=(rank, heads * dim))
    if max(beta_offset + heads, low_offset + (rank or heads), channels) > ld:
        raise KernelError("delta_prepare: a column block lies outside the projection")
    dev = proj.device
    q = torch.empty((n, qk_heads * dim), dtype=torch.float32, device=dev)
    k = torch.empty_like(q)
    v = torch.empty((n, heads * vdim), dtype=torch.float32, device=dev)
    g = torch.empty((n, decays), dtype=torch.float32, device=dev)
    beta = torch.empty((n, heads), dtype=torch.float32, device=dev)
    call("b200_delta_prepare", ptr(proj), ld, beta_offset, low_offset, rank, ptr(taps), ntaps, ptr(conv_state), ptr(a_log),
         ptr(dt_bias), ptr(a_up), ptr(q), ptr(k), ptr(v), ptr(g), ptr(beta), ptr(q_start), ptr(slots), ptr(token_entry),
         n, heads, qk_heads, dim, vdim, float(unit_eps), float(q_scale), tag(proj.dtype), stream_ptr())
    return q, k, v, g, beta


def conv_state_update(proj: torch.Tensor, conv_state: torch.Tensor, q_start: torch.Tensor, slots: torch.Tensor) -> None:
    """After a step: every entry's slot keeps the last ``taps - 1`` inputs of its sequence (columns ``0 .. channels-1``
    of ``proj``), oldest first; a step shorter than that keeps the tail of what the slot held."""

    require(proj, "proj", dims=2)
    require(conv_state, "conv_state", dtype=torch.float32, dims=3)
    entries = q_start.shape[0] - 1
    call("b200_conv_state_update", ptr(proj), proj.shape[1], ptr(conv_state), conv_state.shape[2], conv_state.shape[1] + 1,
         ptr(q_start), ptr(slots), entries, tag(proj.dtype), stream_ptr())


def group_norm_gate(x: torch.Tensor, weight: torch.Tensor | None, eps: float, gate_in: torch.Tensor, *, gate_offset: int = 0,
                    gate_up: torch.Tensor | None = None, out_dtype: torch.dtype, group: int | None = None, act: str = "sigmoid",
                    divisor: "tuple[torch.Tensor, torch.Tensor, float] | None" = None) -> torch.Tensor:
    """``x`` float32 ``[N, width]`` in groups of ``group`` columns (default ``len(weight)``): each group divided by its root mean
    square, times ``weight`` (one group's, or ``[width]``; ``None``: no weight, ``group`` is given), times ``sigmoid(logit)`` or ``silu(logit)`` (``act``).  ``divisor =
    (den, floor, e)``: before that, each group divided by ``max(|den|, floor) + e`` with its own numbers (float32 ``[N, width /
    group]`` each).  The logits are columns ``gate_offset ..`` of ``gate_in`` (``width`` of
    them), or, with ``gate_up`` ``[rank, width]`` (a low-rank map's weight transposed),
    ``gate_in[:, gate_offset : gate_offset + rank] @ gate_up``."""

    require(x, "x", dtype=torch.float32, dims=2)
    n, width = x.shape
    if weight is not None:
        require(weight, "weight", dtype=torch.float32, dims=1)
        group = weight.shape[0] if group is None else group
    if not group or group < 0 or width % group or (weight is not None and weight.shape[0] not in (group, width)):
        raise KernelError(f"width {width} is not a multiple of the group size {group}, or the weight has another number of entries")
    if act not in ("sigmoid", "silu"):
        raise KernelError(f"unknown gate {act!r}")
    den = floor = None
    den_eps = 0.0
    if divisor is not None:
        den, floor, den_eps = divisor
        require(den, "divisor", dtype=torch.float32, shape=(n, width // group))
        require(floor, "divisor floor", dtype=torch.float32, shape=(n, width // group))
    require(gate_in, "gate_in", dtype=out_dtype, dims=2)
    rank = 0
    if gate_up is not None:
        require(gate_up, "gate_up", dtype=out_dtype, dims=2)
        rank = gate_up.shape[0]
        if gate_up.shape[1] != width:
            raise KernelError(f"gate_up has {gate_up.shape[1]} columns, expected {width}")
    if gate_offset + (rank or width) > gate_in.shape[1]:
        raise KernelError("group_norm_gate: the gate's columns lie outside gate_in")
    out = torch.empty((n, width), dtype=out_dtype, device=x.device)
    gate_ptr = gate_in.data_ptr() + gate_offset * gate_in.element_size()
    call("b200_group_norm_gate", ptr(x), n, width, group, ptr(weight), weight.shape[0] if weight is not None else 0, float(eps), ptr(den), ptr(floor), float(den_eps),
         gate_ptr, gate_in.shape[1], rank, ptr(gate_up), 1 if act == "silu" else 0, ptr(out), tag(out_dtype), stream_ptr())
    return out
