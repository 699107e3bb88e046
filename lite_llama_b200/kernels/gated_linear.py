"""Linear attention with data-dependent gates over ragged steps, and the small ops around it
(csrc/gated_linear_attention.cu).  No reference counterpart: the reference's mixers are softmax attention only."""

from __future__ import annotations

import torch

from ._common import check, counters, float_code, lib, ptr, require_cuda, stream_handle

GATED_UNITS = {"silu": 0, "clamped": 1, "gelu_tanh": 2}
GATED_LINEAR_MODES = {"forget_gate": 0, "delta_rule": 1}


@torch.no_grad()
def gated_linear_scan(mode: str, state: torch.Tensor, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, seq_start,
                      seq_ctx, seq_slot, heads: int, qk_heads: int, dim: int, vdim: int, c0: torch.Tensor,
                      c1: torch.Tensor | None = None, p0: torch.Tensor | None = None, p1: torch.Tensor | None = None,
                      q_scale: float = 1.0, unit_eps: float = 1e-6) -> torch.Tensor:
    """``y [tokens, heads * vdim]`` fp32; ``state [slots, heads, dim, vdim]`` fp32 advanced in place.  ``q``, ``k``,
    ``v``, ``p0``, ``p1`` are column views of projections (row strides kept).

    ``"forget_gate"``: ``f = c0 + (1 - c0) * sigmoid(k)`` per key channel (``c0`` = lower bounds ``[heads * dim]``),
    ``S[d, :] <- f[d] S[d, :] + (1 - f[d]) v``, ``y = S^T silu(q)``.
    ``"delta_rule"``: ``q``, ``k`` ``[tokens, qk_heads * dim]`` become unit vectors (``unit_eps`` inside the root; ``q``
    times ``q_scale``); ``g = exp(-exp(c1) * softplus(p1 + c0))``, ``beta = sigmoid(p0)`` per head;
    ``S <- g S; u = beta (v - S^T k); S <- S + k u^T; y = S^T q``."""
    require_cuda(state, q, k, v, c0, c1, p0, p1)
    if state.dtype != torch.float32 or not state.is_contiguous() or tuple(state.shape[1:]) != (heads, dim, vdim):
        raise ValueError("gated_linear_scan: the memory is a contiguous fp32 [slots, heads, dim, vdim] tensor")
    for t in (q, k, v, p0, p1):
        if t is not None and (t.stride(-1) != 1 or t.dtype != q.dtype):
            raise ValueError("gated_linear_scan: the inputs are column views of one dtype")
    tokens = q.shape[0]
    y = torch.empty((tokens, heads * vdim), dtype=torch.float32, device=q.device)
    check(lib().b2l_gated_linear_scan(y.data_ptr(), state.data_ptr(), q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0),
                                      v.data_ptr(), v.stride(0), ptr(p0), p0.stride(0) if p0 is not None else 0, ptr(p1),
                                      p1.stride(0) if p1 is not None else 0, c0.data_ptr(), ptr(c1), seq_start.data_ptr(),
                                      seq_ctx.data_ptr(), seq_slot.data_ptr(), seq_ctx.numel(), heads, qk_heads, dim,
                                      vdim, float(q_scale), float(unit_eps), GATED_LINEAR_MODES[mode],
                                      float_code(q, "q"), stream_handle()))
    return y


MLSTM_CHUNK = 64


def mlstm_head_floats(dim: int, vdim: int) -> int:
    """Floats of one head's state block ``[S: dim x vdim | n: dim | m]``, padded to 16 bytes (the layout of
    csrc/mlstm.cu; ``b2l_mlstm_head_floats``)."""
    return -(-(dim * vdim + dim + 1) // 4) * 4


@torch.no_grad()
def mlstm(state: torch.Tensor, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, zi: torch.Tensor, zf: torch.Tensor,
          bias_i: torch.Tensor, bias_f: torch.Tensor, batch, heads: int, dim: int, vdim: int, gate_cap: float,
          q_scale: float) -> torch.Tensor:
    """Matrix memory with exponential gates over a ragged step: ``y [tokens, heads * vdim]`` fp32; ``state [slots, heads,
    mlstm_head_floats(dim, vdim)]`` fp32 advanced in place.  ``q``, ``k``, ``v`` and the gate logits ``zi``, ``zf
    [tokens, heads]`` are column views of a projection; ``i = cap tanh((zi + bias_i) / cap)``,
    ``f = logsigmoid(cap tanh((zf + bias_f) / cap))``, ``m' = max(f + m, i)``,
    ``S <- e^(f + m - m') S + e^(i - m') k v^T``, ``n`` likewise,
    ``y = S^T q / (max(|n . q|, e^(-m')) + 1e-6)`` with ``q`` times ``q_scale``.  Portions of 16-bit steps that bring at
    least a quarter of a chunk run chunk by chunk on the tensor cores (``dim <= 128``), everything else token by token."""
    require_cuda(state, q, k, v, zi, zf, bias_i, bias_f)
    if state.dtype != torch.float32 or not state.is_contiguous() or state.shape[1:] != (heads, mlstm_head_floats(dim, vdim)):
        raise ValueError("mlstm: the state is a contiguous fp32 [slots, heads, mlstm_head_floats] tensor")
    for t in (q, k, v, zi, zf):
        if t.stride(-1) != 1 or t.dtype != q.dtype:
            raise ValueError("mlstm: the inputs are column views of one dtype")
    if bias_i.dtype != q.dtype or bias_f.dtype != q.dtype:
        raise ValueError("mlstm: gate biases in the activation dtype")
    y = torch.empty((q.shape[0], heads * vdim), dtype=torch.float32, device=q.device)
    cnt = counters(q.device)

    def run(seq_list, count: int, chunked: int) -> None:
        check(lib().b2l_mlstm(y.data_ptr(), state.data_ptr(), q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0),
                              v.data_ptr(), v.stride(0), zi.data_ptr(), zi.stride(0), zf.data_ptr(), zf.stride(0),
                              bias_i.data_ptr(), bias_f.data_ptr(), batch.seq_start.data_ptr(), batch.seq_ctx.data_ptr(),
                              batch.seq_slot.data_ptr(), ptr(seq_list), count, heads, dim, vdim, float(q_scale),
                              float(gate_cap), cnt.data_ptr(), cnt.numel(), chunked, float_code(q, "q"), stream_handle()))

    if q.dtype != torch.float32 and dim <= 128 and batch.max_portion >= MLSTM_CHUNK // 4:
        run(batch.portion_list, batch.num_portions, 1)
        if batch.num_singles:
            run(batch.single_list, batch.num_singles, 0)
    else:
        run(None, batch.num_seqs, 0)
    return y


@torch.no_grad()
def head_norm_gate(y: torch.Tensor, weight: torch.Tensor, heads: int, eps: float,
                   gate: torch.Tensor | None = None, gate_form: str = "silu") -> torch.Tensor:
    """``unit_rms(y[t, h, :]) * weight * silu(gate[t, h, :])`` per head (``gate=None``: no gate; ``gate_form="sigmoid"``:
    its sigmoid); ``y`` fp32 ``[tokens, heads * vdim]``, ``weight [vdim]`` shared by the heads or ``[heads * vdim]``,
    output in ``weight``'s dtype."""
    require_cuda(y, weight, gate)
    rows, inner = y.shape
    vdim = inner // heads
    if y.dtype != torch.float32 or not y.is_contiguous() or weight.numel() not in (vdim, inner) or heads * vdim != inner or \
            gate_form not in ("silu", "sigmoid") or (gate is not None and (gate.stride(-1) != 1 or gate.dtype != weight.dtype)):
        raise ValueError("head_norm_gate: bad layout")
    out = torch.empty((rows, inner), dtype=weight.dtype, device=y.device)
    check(lib().b2l_head_norm_gate(out.data_ptr(), y.data_ptr(), ptr(gate), gate.stride(0) if gate is not None else 0,
                                   weight.data_ptr(), rows, heads, vdim, float(eps), 1 if gate_form == "sigmoid" else 0,
                                   1 if weight.numel() == inner and heads > 1 else 0, float_code(weight, "weight"),
                                   stream_handle()))
    return out


@torch.no_grad()
def head_mix(wide: torch.Tensor, mix: torch.Tensor, heads: int, kv_heads: int, per_call: int, vdim: int) -> torch.Tensor:
    """``out[t, h, :] = sum_g mix[h, g] * wide[t, g, kv(h), :]`` for ``wide [tokens, calls, heads, per_call, vdim]``
    (contiguous), where ``wide[t, c // per_call, g, c % per_call]`` is query head g's softmax weights applied to kv head
    c's values: mixing the heads' attention weights after the softmax equals mixing these outputs."""
    require_cuda(wide, mix)
    rows = wide.shape[0]
    if not wide.is_contiguous() or wide.numel() != rows * heads * kv_heads * vdim or mix.numel() != heads * heads or \
            mix.dtype != wide.dtype or not mix.is_contiguous():
        raise ValueError("head_mix: bad layout")
    out = torch.empty((rows, heads * vdim), dtype=wide.dtype, device=wide.device)
    check(lib().b2l_head_mix(out.data_ptr(), wide.data_ptr(), heads * kv_heads * vdim, mix.data_ptr(), rows, heads, kv_heads,
                             per_call, vdim, float_code(wide, "wide"), stream_handle()))
    return out


@torch.no_grad()
def swiglu_scaled(gate: torch.Tensor, up: torch.Tensor, in_scale: torch.Tensor | None = None,
                  out_logit: torch.Tensor | None = None, form: str = "silu", limit: float = 0.0,
                  alpha: float = 1.702) -> torch.Tensor:
    """``silu(s * gate) * (s * up) * sigmoid(z)`` with one fp32 factor ``s = in_scale[r]`` and one logit
    ``z = out_logit[r, 0]`` per row (both optional).  A factor on a gated unit's INPUT passes through its two linear
    maps, so it is applied here, between the products and the activation.  ``form="clamped"``: the unit is
    ``g' sigmoid(alpha g') (u' + 1)`` with ``g' = min(g, limit)``, ``u' = clamp(u, -limit, limit)`` instead;
    ``form="gelu_tanh"``: ``gelu(g) * u`` with the tanh form of GELU."""
    require_cuda(gate, up, in_scale, out_logit)
    rows, n = gate.shape
    if up.shape != gate.shape or gate.stride(-1) != 1 or up.stride(-1) != 1 or up.dtype != gate.dtype or \
            (in_scale is not None and (in_scale.dtype != torch.float32 or in_scale.numel() != rows or not in_scale.is_contiguous())) or \
            (out_logit is not None and (out_logit.dtype != gate.dtype or out_logit.shape[0] != rows)):
        raise ValueError("swiglu_scaled: bad layout")
    out = torch.empty((rows, n), dtype=gate.dtype, device=gate.device)
    check(lib().b2l_swiglu_scaled(out.data_ptr(), out.stride(0), gate.data_ptr(), gate.stride(0), up.data_ptr(),
                                  up.stride(0), ptr(in_scale), ptr(out_logit),
                                  out_logit.stride(0) if out_logit is not None else 0, rows, n, GATED_UNITS[form],
                                  float(limit), float(alpha), float_code(gate, "gate"), stream_handle()))
    return out
