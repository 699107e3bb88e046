"""A residual kept as several streams (hyper-connections) and the input convolution of single-token steps
(csrc/hyper_stream.cu).  No reference counterpart: the reference keeps one 16-bit residual
(lite_llama/models/base.py:299-319)."""

from __future__ import annotations

import torch

from ._common import check, float_code, lib, ptr, require_cuda, stream_handle

MAX_STREAMS = 8


def _conv_args(conv, h: torch.Tensor):
    """``conv = (weight [n, taps], tail [slots, taps - 1, n], seq_ctx, seq_slot)`` of a step in which every token is a
    sequence of its own -> (pointers, the convolved copy of ``h``)."""
    if conv is None:
        return (None, None, None, None, None, 0), None
    weight, tail, seq_ctx, seq_slot = conv
    require_cuda(weight, tail, seq_ctx, seq_slot)
    if weight.dtype != h.dtype or weight.shape[0] != h.shape[1] or not weight.is_contiguous() or seq_ctx.numel() != h.shape[0]:
        raise ValueError("stream kernels: bad convolution layout")
    hc = torch.empty_like(h)
    return (weight.data_ptr(), ptr(tail), hc.data_ptr(), seq_ctx.data_ptr(), seq_slot.data_ptr(), weight.shape[1]), hc


@torch.no_grad()
def stream_embed(tokens: torch.Tensor, embed: torch.Tensor, embed_weight: torch.Tensor, streams: int, read_in: torch.Tensor,
                 weight: torch.Tensor, eps: float, conv=None):
    """All streams = ``unit_rms(embed[token]) * embed_weight``; then a read ``h = unit_rms(sum_s read_in[s] x_s) * weight``.
    Returns ``(x [tokens, streams, n] fp32, h, hc)``; ``hc`` (``None`` without ``conv``) is ``h`` plus its causal
    convolution, see ``_conv_args``."""
    require_cuda(tokens, embed, embed_weight, read_in, weight)
    if tokens.dtype != torch.int32 or read_in.dtype != torch.float32 or read_in.numel() != streams:
        raise ValueError("stream_embed: int32 tokens, fp32 read coefficients")
    rows, n = tokens.numel(), embed.shape[1]
    x = torch.empty((rows, streams, n), dtype=torch.float32, device=embed.device)
    h = torch.empty((rows, n), dtype=embed.dtype, device=embed.device)
    (cw, tail, hcp, cx, sl, taps), hc = _conv_args(conv, h)
    check(lib().b2l_stream_embed(x.data_ptr(), tokens.data_ptr(), embed.data_ptr(), embed_weight.data_ptr(), embed.shape[0],
                                 read_in.data_ptr(), weight.data_ptr(), h.data_ptr(), cw, tail, hcp, cx, sl, taps, rows,
                                 streams, n, float(eps), float_code(embed, "embed"), stream_handle()))
    return x, h, hc


@torch.no_grad()
def stream_mix(x: torch.Tensor, y: torch.Tensor, coef: torch.Tensor, read_in: torch.Tensor, weight: torch.Tensor, eps: float,
               addend: torch.Tensor | None = None, gate: torch.Tensor | None = None, gate_bias: torch.Tensor | None = None,
               rows: torch.Tensor | None = None, conv=None):
    """A sublayer's write into the streams ``x [tokens, streams, n]`` (fp32, in place) and the next sublayer's read, one
    launch: ``x_t <- sum_s mix[s, t] x_s + out[t] y'`` with ``coef = [out: streams | mix: streams * streams (from, to)]``
    (fp32), ``y' = (y + addend) * sigmoid(gate + gate_bias)`` (``y [tokens, terms, n]``: the sum over the terms;
    ``addend`` / ``gate`` optional), then ``h = unit_rms(sum_s read_in[s] x_s) * weight``.  Returns ``(h, hc)``, ``hc`` as in
    ``stream_embed``.  ``rows``: only these tokens are read (``h`` compact) and ``x`` stays as it is."""
    require_cuda(x, y, coef, read_in, weight, addend, gate, gate_bias, rows)
    tokens, streams, n = x.shape
    terms = y.shape[1] if y.dim() == 3 else 1
    y2d = y.reshape(tokens * terms, n)
    if x.dtype != torch.float32 or not x.is_contiguous() or y2d.stride(-1) != 1 or coef.numel() != streams * (streams + 1) or \
            read_in.numel() != streams or coef.dtype != torch.float32 or read_in.dtype != torch.float32:
        raise ValueError("stream_mix: bad stream layout")
    for t in (addend, gate):
        if t is not None and (t.shape != (tokens, n) or t.stride(-1) != 1 or t.dtype != y.dtype):
            raise ValueError("stream_mix: addend and gate are [tokens, n] in y's dtype")
    if weight.dtype != y.dtype or (gate is None) != (gate_bias is None) or (rows is not None and (rows.dtype != torch.int32 or conv)):
        raise ValueError("stream_mix: bad norm weight, gate or row list")
    count = tokens if rows is None else rows.numel()
    h = torch.empty((count, n), dtype=y.dtype, device=x.device)
    (cw, tail, hcp, cx, sl, taps), hc = _conv_args(conv, h)
    check(lib().b2l_stream_mix(x.data_ptr(), y2d.data_ptr(), y2d.stride(0), terms, ptr(addend),
                               addend.stride(0) if addend is not None else 0, ptr(gate),
                               gate.stride(0) if gate is not None else 0, ptr(gate_bias), coef.data_ptr(),
                               read_in.data_ptr(), weight.data_ptr(), h.data_ptr(), ptr(rows), cw, tail, hcp, cx, sl, taps,
                               count, streams, n, float(eps), float_code(y, "y"), stream_handle()))
    return h, hc
