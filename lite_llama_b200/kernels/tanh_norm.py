"""Residual of designs whose sublayers read an element-wise norm, ``tanh(alpha x) * w + b``, and add their result as it is
(csrc/tanh_norm_stream.cu): one pass per sublayer boundary adds the finished sublayer (or sums its expert terms, identity
experts among them), what a loop adds where a pass starts, and hands out the next sublayer's input.  The reference's norms
are row statistics in front of a 16-bit residual (lite_llama/kernels/skip_rmsnorm.py)."""

from __future__ import annotations

import torch

from ._common import check, float_code, lib, ptr, require_cuda, stream_handle


@torch.no_grad()
def tanh_norm_stream(residual: torch.Tensor, norm: tuple[torch.Tensor, torch.Tensor, torch.Tensor] | None = None, *,
                     y: torch.Tensor | None = None, routed: tuple[torch.Tensor, torch.Tensor, int, torch.Tensor] | None = None,
                     addend: torch.Tensor | None = None, embedding: tuple[torch.Tensor, torch.Tensor, float] | None = None,
                     step: torch.Tensor | None = None, first: bool = False, rows: torch.Tensor | None = None) -> torch.Tensor | None:
    """In place on the fp32 ``residual [T, n]``: ``+ y [T, n]`` (``first``: starts from zero, there is no ``y``), ``+
    scale * table[tokens]`` for ``embedding = (tokens, table, scale)``, ``+ step [n]``; returns ``tanh(alpha v) * w + b`` for
    ``norm = (w, b, alpha)`` in their dtype (``None`` without a norm).  ``routed = (ids, weights, experts, x)``: ``y`` is
    ``[T, top, n]``, the weighted outputs of the chosen experts ``ids [T, top]``; ids from ``experts`` on stand for
    ``weights * x``; ``addend [T, n]`` joins their sum.  ``rows``: only these tokens are read and normed, the residual is
    not written."""
    require_cuda(residual, y, addend, step, rows)
    T, n = residual.shape
    if residual.dtype != torch.float32 or not residual.is_contiguous():
        raise ValueError("tanh_norm_stream: the residual is a contiguous fp32 tensor")
    w, b, alpha = norm if norm is not None else (None, None, None)
    ids, weights, experts, x = routed if routed is not None else (None, None, 0, None)
    tokens, table, scale = embedding if embedding is not None else (None, None, 0.0)
    tensors = [t for t in (y, addend, step, table, w, b, alpha, x) if t is not None]
    ref = tensors[0] if tensors else None
    if ref is None or any(t.dtype != ref.dtype for t in tensors):
        raise ValueError("tanh_norm_stream: operands of one dtype")
    if norm is not None and (w.numel() != n or b.numel() != n or alpha.numel() != 1):
        raise ValueError("tanh_norm_stream: norm weight and shift are [n], alpha is one number")
    top = 0
    if y is not None:
        if y.stride(-1) != 1 or y.shape[0] != T or y.shape[-1] != n or (routed is None) != (y.dim() == 2):
            raise ValueError("tanh_norm_stream: bad layout of the sublayer's result")
        if routed is not None:
            top = y.shape[1]
            if ids.shape != (T, top) or weights.shape != (T, top) or ids.dtype != torch.int32 or weights.dtype != torch.float32 or \
                    not (ids.is_contiguous() and weights.is_contiguous() and y.is_contiguous()) or x.shape != (T, n) or x.stride(-1) != 1:
                raise ValueError("tanh_norm_stream: routed results are contiguous, ids int32, weights fp32")
    if (addend is not None and (addend.shape != (T, n) or not addend.is_contiguous())) or \
            (step is not None and step.numel() != n) or (tokens is not None and (tokens.dtype != torch.int32 or table.shape[1] != n)) or \
            (rows is not None and rows.dtype != torch.int32):
        raise ValueError("tanh_norm_stream: bad operand")
    count = T if rows is None else rows.numel()
    act = torch.empty((count, n), dtype=ref.dtype, device=residual.device) if norm is not None else None
    check(lib().b2l_tanh_norm_stream(residual.data_ptr(), ptr(act), ptr(y), y.stride(-2) if y is not None else 0, top, ptr(ids),
                                     ptr(weights), int(experts), ptr(x), x.stride(0) if x is not None else 0, ptr(addend),
                                     ptr(tokens), ptr(table), table.shape[0] if table is not None else 0, float(scale),
                                     ptr(step), 1 if first else 0, ptr(alpha), ptr(w), ptr(b), ptr(rows), count, n,
                                     float_code(ref, "operands"), stream_handle()))
    return act
