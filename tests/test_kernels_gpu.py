"""Parity tests proper: the sm_100a CUDA kernels (through the C ABI / ctypes shims) against
(1) the golden outputs recorded from the reference's own Triton kernels and (2) the CPU oracle on
seeded random inputs, on the case lists of the reference's tests/kernels/*.py, plus the
reference-free invariants those tests use.

Tolerances (stated per op, always tighter than or equal to the reference's own test tolerances):
  integer / index results ......... bit-exact
  norm / swiglu / rope ............ 2 fp16 ulp (rtol 2e-3, atol 1e-3 [rope: 4e-3 for |x| up to 8])
  attention ....................... rtol 2e-3, atol 2e-3   (reference tests: 1e-2 .. 2e-2)
  GEMMs (dense, w4a16, w8a16, w8a8) rtol 2e-3, atol 2e-3 on O(1) outputs (reference: 1e-2 .. 1e-1)
"""

from __future__ import annotations

import math
import os

import pytest
import torch

from b2l_testutil import load_golden, to_cuda
from oracle import ops

pytestmark = [pytest.mark.gpu, pytest.mark.timeout(180)]

LOG2E = 1.4426950408889634
TOL = dict(rtol=2e-3, atol=1e-3)
ATT_TOL = dict(rtol=2e-3, atol=2e-3)
GEMM_TOL = dict(rtol=2e-3, atol=2e-3)


def K():
    import lite_llama_b200.kernels as k

    return k


def close(actual, expected, **tol):
    torch.testing.assert_close(actual.float().cpu(), expected.float().cpu(), **(tol or TOL))


# --------------------------------------------------------------------------- #
# skip_rmsnorm
# --------------------------------------------------------------------------- #
def test_skip_rmsnorm_golden():
    for c in load_golden("skip_rmsnorm")["cases"]:
        g = to_cuda(c)
        res = None if g["residual"] is None else g["residual"].clone()
        y, r = K().skip_rmsnorm(g["x"].clone(), res, g["weight"], g["eps"])
        close(y, c["y"])
        if c["residual"] is not None:
            assert torch.equal(r.cpu(), c["residual_out"])


@pytest.mark.parametrize("shape", [(1, 1, 64), (2, 5, 896), (3, 7, 4096), (4, 1, 3584), (2, 3, 100), (1, 2, 8192)])
@pytest.mark.parametrize("dtype", [torch.float16, torch.bfloat16])
def test_skip_rmsnorm_matches_oracle(shape, dtype):
    x = torch.randn(shape, device="cuda", dtype=dtype)
    r = torch.randn(shape, device="cuda", dtype=dtype)
    w = torch.randn(shape[-1], device="cuda", dtype=dtype)
    y_ref, r_ref = ops.skip_rmsnorm(x.cpu(), r.cpu(), w.cpu(), 1e-5)
    r_in = r.clone()
    y, r_out = K().skip_rmsnorm(x, r_in, w, 1e-5)
    tol = TOL if dtype == torch.float16 else dict(rtol=1.6e-2, atol=8e-3)
    close(y, y_ref, **tol)
    assert torch.equal(r_out.cpu(), r_ref)
    assert r_out.data_ptr() == r_in.data_ptr(), "residual must be updated in place and returned aliased"
    y2, x_back = K().skip_rmsnorm(x, None, w, 1e-5)
    close(y2, ops.rmsnorm(x.cpu(), w.cpu(), 1e-5), **tol)
    assert x_back.data_ptr() == x.data_ptr()


def test_skip_rmsnorm_wide_unaligned_rows_with_residual():
    """Rows wider than 4096 whose length is not a multiple of 8 take the two-pass warp kernel, residual included
    (that combination used to be rejected)."""
    x = torch.randn(3, 4100 + 3, device="cuda", dtype=torch.float16)
    res = torch.randn_like(x)
    w = torch.randn(x.shape[-1], device="cuda", dtype=torch.float16)
    y, r = K().skip_rmsnorm(x, res.clone(), w, 1e-5)
    yr, rr = ops.skip_rmsnorm(x.cpu(), res.cpu(), w.cpu(), 1e-5)
    close(y.cpu(), yr, rtol=2e-3, atol=2e-3)
    close(r.cpu(), rr, rtol=1e-3, atol=1e-3)


def test_skip_rmsnorm_per_head_layout():
    # the Qwen3 q/k-norm call: [tokens, heads, head_dim] normalised over head_dim (models/base.py:222-225)
    x = torch.randn(7, 14, 128, device="cuda", dtype=torch.float16)
    w = torch.randn(128, device="cuda", dtype=torch.float16)
    y, _ = K().skip_rmsnorm(x, None, w, 1e-6)
    close(y, ops.rmsnorm(x.cpu(), w.cpu(), 1e-6))


def test_skip_rmsnorm_known_answer():
    x = torch.full((2, 3, 64), 2.0, device="cuda", dtype=torch.float16)
    r = torch.full((2, 3, 64), 3.0, device="cuda", dtype=torch.float16)
    w = (torch.arange(64, device="cuda") / 64).half()
    y, res = K().skip_rmsnorm(x, r, w, 1e-6)
    close(y, w.expand(2, 3, 64))
    assert (res == 5).all()


# --------------------------------------------------------------------------- #
# swiglu / rope
# --------------------------------------------------------------------------- #
def test_swiglu_golden_and_oracle():
    for c in load_golden("swiglu")["cases"]:
        g = to_cuda(c)
        close(K().swiglu_forward(g["a"], g["b"]), c["out"])
    for shape in [(1, 1, 14336), (2, 3, 18944), (5, 100)]:
        a = torch.randn(shape, device="cuda", dtype=torch.float16) * 3
        b = torch.randn(shape, device="cuda", dtype=torch.float16)
        close(K().swiglu_forward(a, b), ops.swiglu(a.cpu(), b.cpu()))
    z = torch.zeros(4, 256, device="cuda", dtype=torch.float16)
    assert (K().swiglu_forward(z, torch.randn_like(z)) == 0).all(), "zero gate must give zero"


def test_rope_golden_bit_exact_where_the_interpreter_agrees():
    # the kernel contracts mul+fma exactly like Triton's sm_100 codegen; the interpreter rounds each
    # op, so allow 1 ulp at |x| < 8 against the golden and 2 ulp against the fp32 oracle
    for c in load_golden("rope")["cases"]:
        g = to_cuda(c)
        q, k = K().rope_emb_forward(g["q"].clone(), g["k"].clone(), g["cos"], g["sin"], c["batch"], c["seq"])
        close(q, c["q_out"], rtol=2e-3, atol=4e-3)
        close(k, c["k_out"], rtol=2e-3, atol=4e-3)


@pytest.mark.parametrize("hd", [32, 64, 128])
def test_rope_matches_oracle_and_is_in_place(hd):
    b, s, hq, hk = 2, 9, 8, 2
    q = torch.randn(b * s, hq, hd, device="cuda", dtype=torch.float16)
    k = torch.randn(b * s, hk, hd, device="cuda", dtype=torch.float16)
    ang = torch.rand(b, s, hd // 2, device="cuda") * 6.28
    cos = torch.cat([ang.cos(), ang.cos()], -1).half()
    sin = torch.cat([ang.sin(), ang.sin()], -1).half()
    q_ref = ops.rope_half_split(q.cpu(), cos.cpu(), sin.cpu(), b, s)
    k_ref = ops.rope_half_split(k.cpu(), cos.cpu(), sin.cpu(), b, s)
    q_in, k_in = q.clone(), k.clone()
    qo, ko = K().rope_emb_forward(q_in, k_in, cos, sin, b, s)
    close(qo, q_ref, rtol=2e-3, atol=4e-3)
    close(ko, k_ref, rtol=2e-3, atol=4e-3)
    assert qo.data_ptr() == q_in.data_ptr() and ko.data_ptr() == k_in.data_ptr()
    # zero angle is the identity (tests/kernels/test_rope_emb.py:80-96)
    one, zero = torch.ones_like(cos), torch.zeros_like(sin)
    q2, _ = K().rope_emb_forward(q.clone(), k.clone(), one, zero, b, s)
    assert torch.equal(q2, q)
    # rotation preserves the pairwise norm
    n0 = (q[..., : hd // 2].float() ** 2 + q[..., hd // 2 :].float() ** 2)
    n1 = (qo[..., : hd // 2].float() ** 2 + qo[..., hd // 2 :].float() ** 2)
    torch.testing.assert_close(n0, n1, rtol=1e-2, atol=1e-2)


# --------------------------------------------------------------------------- #
# KV cache ops (bit-exact)
# --------------------------------------------------------------------------- #
def test_kv_ops_golden():
    g = load_golden("kv_ops")
    c = to_cuda(g)
    buf = c["buffer"].clone()
    K().update_kv_buffer(c["values"], c["select"], buf)
    assert torch.equal(buf.cpu(), g["buffer_out"])
    table = c["table"].clone()
    K().update_kv_index(table, c["b_req_idx"], c["b_seq_len"], c["select_index"])
    assert torch.equal(table.cpu(), g["table_out"])


@pytest.mark.parametrize("idx_dtype", [torch.int32, torch.int64])
def test_update_kv_buffer_strided_pool_and_untouched_rows(idx_dtype):
    hkv, d, tokens, pool_rows = 4, 128, 37, 300
    pool = torch.randn(pool_rows, 2 * hkv, d, device="cuda", dtype=torch.float16)
    before = pool.clone()
    vals = torch.randn(tokens, 2 * hkv, d, device="cuda", dtype=torch.float16)
    sel = torch.randperm(pool_rows, device="cuda")[:tokens].to(idx_dtype if idx_dtype == torch.int64 else torch.int32)
    K().update_kv_buffer(vals, sel, pool)
    expect = ops.update_kv_buffer(vals.cpu(), sel.cpu(), before.cpu())
    assert torch.equal(pool.cpu(), expect)
    # split K/V sources written without torch.cat
    pool2 = before.clone()
    xkv = torch.randn(tokens, 2 * hkv * d, device="cuda", dtype=torch.float16)
    xk, xv = torch.split(xkv, hkv * d, dim=-1)
    K().update_kv_buffer_split(xk.view(tokens, hkv, d), xv.view(tokens, hkv, d), sel, pool2)
    expect2 = ops.update_kv_buffer(xkv.view(tokens, 2 * hkv, d).cpu(), sel.cpu(), before.cpu())
    assert torch.equal(pool2.cpu(), expect2)


@pytest.mark.parametrize("dt", [torch.int32, torch.int64])
def test_update_kv_index_both_index_widths(dt):
    table = torch.zeros(8, 64, dtype=torch.int32, device="cuda")
    req = torch.tensor([5, 0, 7, 2], device="cuda", dtype=dt)
    lens = torch.tensor([1, 64, 33, 2], device="cuda", dtype=dt)
    sel = torch.tensor([11, 22, 33, 44], device="cuda", dtype=torch.int32)
    K().update_kv_index(table, req, lens, sel)
    expect = ops.update_kv_index(torch.zeros(8, 64, dtype=torch.int32), req.cpu(), lens.cpu(), sel.cpu())
    assert torch.equal(table.cpu(), expect)


# --------------------------------------------------------------------------- #
# flash_decoding
# --------------------------------------------------------------------------- #
_MAX_TOKENS = 2048


def _decode_case(seq_lens, hq, hkv, d, *, scattered=False, req_idx=None, dtype=torch.float16, idx=torch.int32,
                 fused_pool=False):
    q = torch.randn(len(seq_lens), hq, d, device="cuda", dtype=dtype) * 0.3
    width = max(seq_lens)
    nslots = len(seq_lens)
    rows = max(_MAX_TOKENS, nslots * width)
    if fused_pool:
        pool = torch.randn(rows, 2 * hkv, d, device="cuda", dtype=dtype)
        kc, vc = pool[:, :hkv], pool[:, hkv:]
    else:
        kc = torch.randn(rows, hkv, d, device="cuda", dtype=dtype)
        vc = torch.randn(rows, hkv, d, device="cuda", dtype=dtype)
    table = torch.zeros(nslots, width, dtype=torch.int32, device="cuda")
    if scattered:
        perm = torch.randperm(rows, device="cuda").to(torch.int32)
        for i in range(nslots):
            table[i] = perm[i * width : (i + 1) * width]
    else:
        for i in range(nslots):
            table[i] = torch.arange(i * width, (i + 1) * width, dtype=torch.int32, device="cuda")
    b_seq = torch.tensor(seq_lens, dtype=idx, device="cuda")
    b_req = torch.arange(nslots, dtype=idx, device="cuda") if req_idx is None else torch.tensor(req_idx, dtype=idx, device="cuda")
    scale = 1.0 / math.sqrt(d)
    out = K().flash_decoding(q, kc, vc, scale, table, b_req, b_seq, width)
    ref = ops.paged_decode_attention(q.cpu(), kc.cpu(), vc.cpu(), table.cpu(), b_req.cpu(), b_seq.cpu(), scale)
    return out, ref


def test_flash_decoding_golden():
    for c in load_golden("flash_decoding")["cases"]:
        g = to_cuda(c)
        out = K().flash_decoding(g["q"], g["k_cache"], g["v_cache"], c["scale"], g["table"], g["b_req_idx"],
                                 g["b_seq_len"], c["max_len"])
        close(out, c["out"], **ATT_TOL)


@pytest.mark.parametrize("seq_lens", [[1], [15], [16], [17], [63], [64], [65], [128], [129], [255], [256], [257], [1000]])
def test_flash_decoding_boundaries(seq_lens):
    out, ref = _decode_case(seq_lens, 4, 4, 64)
    assert torch.isfinite(out).all()
    close(out, ref, **ATT_TOL)


@pytest.mark.parametrize("seq_lens", [[32, 32], [1, 200], [17, 129, 64, 3], [700, 5, 1300, 64]])
def test_flash_decoding_ragged(seq_lens):
    out, ref = _decode_case(seq_lens, 4, 2, 64)
    close(out, ref, **ATT_TOL)


@pytest.mark.parametrize("hq,hkv", [(4, 4), (8, 2), (14, 2), (8, 1), (32, 8), (28, 4), (32, 1)])
def test_flash_decoding_gqa_ratios(hq, hkv):
    out, ref = _decode_case([48, 130], hq, hkv, 64)
    close(out, ref, **ATT_TOL)


@pytest.mark.parametrize("d", [32, 64, 128])
@pytest.mark.parametrize("dtype", [torch.float16, torch.bfloat16])
def test_flash_decoding_head_dims_and_dtypes(d, dtype):
    out, ref = _decode_case([40, 150], 4, 2, d, dtype=dtype)
    tol = ATT_TOL if dtype == torch.float16 else dict(rtol=1.6e-2, atol=1.6e-2)
    close(out, ref, **tol)


@pytest.mark.parametrize("seq_lens", [[64], [33, 130]])
def test_flash_decoding_scattered_rows(seq_lens):
    out, ref = _decode_case(seq_lens, 4, 2, 64, scattered=True)
    close(out, ref, **ATT_TOL)


def test_flash_decoding_slot_indirection_and_int64_indices():
    out, ref = _decode_case([40, 24, 61], 8, 8, 64, req_idx=[2, 1, 0], idx=torch.int64)
    close(out, ref, **ATT_TOL)
    out, ref = _decode_case([33, 33, 33], 4, 2, 64, req_idx=[0, 1, 1])
    close(out, ref, **ATT_TOL)


def test_flash_decoding_on_the_fused_kv_pool_views():
    # the model hands strided views kv[:, :Hkv], kv[:, Hkv:] of one pool (models/base.py:119-123)
    out, ref = _decode_case([100, 300, 7], 32, 8, 128, fused_pool=True)
    close(out, ref, **ATT_TOL)


def test_flash_decoding_uniform_values():
    d, n = 64, 150
    q = torch.randn(1, 4, d, device="cuda", dtype=torch.float16) * 0.3
    kc = torch.randn(_MAX_TOKENS, 4, d, device="cuda", dtype=torch.float16)
    vc = torch.full((_MAX_TOKENS, 4, d), 0.25, device="cuda", dtype=torch.float16)
    table = torch.arange(n, dtype=torch.int32, device="cuda").unsqueeze(0)
    out = K().flash_decoding(q, kc, vc, 1 / math.sqrt(d), table, torch.zeros(1, dtype=torch.int32, device="cuda"),
                             torch.tensor([n], dtype=torch.int32, device="cuda"), n)
    close(out, torch.full_like(out, 0.25), **ATT_TOL)


def test_flash_decoding_llama3_shape_long_context():
    # BASELINE shape: B=32, Hq=32, Hkv=8, D=128; ragged contexts up to 2048
    torch.manual_seed(1)
    B, hq, hkv, d, ctx = 8, 32, 8, 128, 2048
    pool_rows = B * ctx
    pool = torch.randn(pool_rows, 2 * hkv, d, device="cuda", dtype=torch.float16)
    kc, vc = pool[:, :hkv], pool[:, hkv:]
    lens = torch.randint(ctx // 2, ctx + 1, (B,))
    table = torch.arange(pool_rows, dtype=torch.int32, device="cuda").view(B, ctx)
    q = torch.randn(B, hq, d, device="cuda", dtype=torch.float16) * 0.3
    b_seq = lens.to(torch.int32).cuda()
    b_req = torch.arange(B, dtype=torch.int32, device="cuda")
    out = K().flash_decoding(q, kc, vc, 1 / math.sqrt(d), table, b_req, b_seq, ctx)
    ref = ops.paged_decode_attention(q.cpu(), kc.cpu(), vc.cpu(), table.cpu(), b_req.cpu(), b_seq.cpu(), 1 / math.sqrt(d))
    close(out, ref, **ATT_TOL)


@pytest.mark.parametrize("m", [1, 32, 64, 200])
def test_w4a16_swiglu_epilogue_is_bit_identical_to_gemm_then_swiglu(m):
    """gate|up rows interleaved at load time + silu(gate) * up in the GEMM epilogue (stream-K fix-up path included:
    N = 1024, K = 512 splits tiles across CTAs) against the unfused path: w4a16 GEMM, then swiglu_forward."""
    from lite_llama_b200.kernels.quantization import interleave_gate_up

    torch.manual_seed(m)
    inter, k = 512, 512
    w = torch.randn(2 * inter, k) * 0.05
    qw, sc, zp = (t.cuda() for t in ops.quantize_int4_groupwise(w, 128))
    x = torch.randn(m, k, device="cuda", dtype=torch.float16)
    gu = K().w4a16_matmul(x, qw, sc, zp, group_size=128)
    want = K().swiglu_forward(gu[:, :inter], gu[:, inter:])
    packed = K().w4a16_pack(interleave_gate_up(qw), interleave_gate_up(sc), interleave_gate_up(zp), group_size=128)
    got = K().w4a16_matmul_packed(x, packed, swiglu=True)
    assert got.shape == (m, inter)
    assert torch.equal(got, want)


def test_rope_kv_write_equals_rope_then_cache_write():
    """The fused launch (rope on q/k where they lie + K|V cache write) against the two-step path the reference takes
    (rope_emb_forward, then torch.cat + update_kv_buffer: models/base.py:76-79,228) -- bit for bit, on the strided
    views of one fused-qkv buffer, prefill rectangle and decode step, scattered cache rows, int32/int64 indices."""
    for (B, S, hq, hkv, d, idx_dtype) in [(3, 5, 8, 2, 64, torch.int32), (32, 1, 32, 8, 128, torch.int64),
                                         (1, 1, 14, 2, 64, torch.int32), (2, 130, 4, 4, 32, torch.int32)]:
        T = B * S
        qkv = torch.randn(T, (hq + 2 * hkv) * d, device="cuda", dtype=torch.float16)
        cos = torch.randn(B, S, d, device="cuda", dtype=torch.float16)
        sin = torch.randn(B, S, d, device="cuda", dtype=torch.float16)
        rows = torch.randperm(4 * T, device="cuda")[:T].to(idx_dtype)
        pool_a = torch.zeros(4 * T, 2 * hkv, d, device="cuda", dtype=torch.float16)
        pool_b = torch.zeros_like(pool_a)

        def views(buf):
            return (buf[:, : hq * d].view(T, hq, d), buf[:, hq * d : (hq + hkv) * d].view(T, hkv, d),
                    buf[:, (hq + hkv) * d :].view(T, hkv, d))

        a, b = qkv.clone(), qkv.clone()
        qa, ka, va = views(a)
        K().rope_emb_inplace(qa, ka, cos, sin, B, S)
        K().update_kv_buffer_split(ka, va, rows, pool_a)
        qb, kb, vb = views(b)
        K().rope_kv_write(qb, kb, vb, cos, sin, rows, pool_b, B, S)
        assert torch.equal(a, b), "rotated q/k differ"
        assert torch.equal(pool_a, pool_b), "cache rows differ"
        ref_q = ops.rope_half_split(views(qkv.cpu())[0], cos.cpu(), sin.cpu(), B, S)
        close(qb.cpu(), ref_q, rtol=2e-3, atol=2e-3)


# --------------------------------------------------------------------------- #
# flash_attention2_no_pad
# --------------------------------------------------------------------------- #
def _prefill_case(seq_lens, hq, hkv, d, dtype=torch.float16, padded_to=None, strided_kv=False):
    if padded_to is None:
        starts = [sum(seq_lens[:i]) for i in range(len(seq_lens))]
        total = sum(seq_lens)
    else:  # the engine's padded rectangle: sequence i starts at i*max_prompt_len (model_runner.py:153-179)
        starts = [i * padded_to for i in range(len(seq_lens))]
        total = padded_to * len(seq_lens)
    q = torch.randn(total, hq, d, device="cuda", dtype=dtype) * 0.3
    if strided_kv:
        xkv = torch.randn(total, 2 * hkv * d, device="cuda", dtype=dtype) * 0.3
        k, v = (t.view(total, hkv, d) for t in torch.split(xkv, hkv * d, dim=-1))
    else:
        k = torch.randn(total, hkv, d, device="cuda", dtype=dtype) * 0.3
        v = torch.randn(total, hkv, d, device="cuda", dtype=dtype) * 0.3
    b_start = torch.tensor(starts, dtype=torch.int32, device="cuda")
    b_len = torch.tensor(seq_lens, dtype=torch.int32, device="cuda")
    scale = 1.0 / math.sqrt(d)
    out = K().flash_attention2_no_pad(q, k, v, scale * LOG2E, b_start, b_len, max(seq_lens))
    ref = ops.varlen_causal_attention(q.cpu(), k.cpu(), v.cpu(), b_start.cpu(), b_len.cpu(), scale)
    valid = torch.zeros(total, dtype=torch.bool)
    for s, n in zip(starts, seq_lens):
        valid[s : s + n] = True
    return out.cpu()[valid], ref[valid], (q, k, v)


def test_flash_attention_nopad_golden():
    for c in load_golden("flash_attention_nopad")["cases"]:
        g = to_cuda(c)
        out = K().flash_attention2_no_pad(g["q"], g["k"], g["v"], c["scale"] * LOG2E, g["b_start_loc"],
                                          g["b_seq_len"], c["max_len"])
        valid = torch.zeros(c["q"].shape[0], dtype=torch.bool)
        for s, n in zip(c["b_start_loc"].tolist(), c["b_seq_len"].tolist()):
            valid[s : s + n] = True
        close(out.cpu()[valid], c["out"][valid], **ATT_TOL)


@pytest.mark.parametrize("seq_lens", [[16], [64], [100], [32, 32], [7, 100, 33], [1, 64], [129, 65, 200], [513]])
def test_flash_attention_nopad_ragged(seq_lens):
    out, ref, _ = _prefill_case(seq_lens, 4, 4, 64)
    close(out, ref, **ATT_TOL)


@pytest.mark.parametrize("hq,hkv", [(4, 4), (8, 2), (14, 2), (8, 1), (32, 8)])
def test_flash_attention_nopad_gqa(hq, hkv):
    out, ref, _ = _prefill_case([48, 24], hq, hkv, 64)
    close(out, ref, **ATT_TOL)


@pytest.mark.parametrize("d", [32, 64, 128])
@pytest.mark.parametrize("dtype", [torch.float16, torch.bfloat16])
def test_flash_attention_nopad_head_dims(d, dtype):
    out, ref, _ = _prefill_case([40, 24], 4, 2, d, dtype=dtype)
    tol = ATT_TOL if dtype == torch.float16 else dict(rtol=1.6e-2, atol=1.6e-2)
    close(out, ref, **tol)


def test_flash_attention_nopad_padded_rectangle_and_strided_kv():
    out, ref, _ = _prefill_case([128, 90, 17], 32, 8, 128, padded_to=128, strided_kv=True)
    close(out, ref, **ATT_TOL)


# head_dim 128 with packed heads runs the tcgen05 kernel (csrc/flash_attention_tc.cu): 128-row query blocks, 128-key
# tiles, S/P/O in tensor memory.  Cases: one partial block, exact block boundaries, several key tiles per block (the
# double-buffered S / O pipeline and all three ring stages wrap), ragged batches, GQA, strided fused-qkv views, bf16.
@pytest.mark.parametrize("seq_lens", [[1], [17], [127], [128], [129], [255, 256, 257], [300, 5, 128], [1024], [2048, 640]])
def test_flash_attention_tc_ragged_d128(seq_lens):
    out, ref, _ = _prefill_case(seq_lens, 8, 2, 128)
    close(out, ref, **ATT_TOL)


@pytest.mark.parametrize("hq,hkv", [(4, 4), (8, 1), (32, 8), (28, 4)])
@pytest.mark.parametrize("dtype", [torch.float16, torch.bfloat16])
def test_flash_attention_tc_gqa_dtypes_d128(hq, hkv, dtype):
    out, ref, _ = _prefill_case([200, 130], hq, hkv, 128, dtype=dtype, strided_kv=True)
    tol = ATT_TOL if dtype == torch.float16 else dict(rtol=1.6e-2, atol=1.6e-2)
    close(out, ref, **tol)


def test_flash_attention_tc_matches_the_mma_sync_kernel_on_the_llama_prefill_shape():
    """BASELINE prefill: 32 sequences x 128 tokens, Llama-3-8B heads, q/k/v as views of one fused-qkv buffer in the
    padded-rectangle layout; the tcgen05 kernel against the oracle and against the mma.sync kernel (B2L_FA_TC=0 path
    is exercised by the head_dim 32/64 cases above)."""
    B, S, hq, hkv, d = 32, 128, 32, 8, 128
    total = B * S
    qkv = torch.randn(total, (hq + 2 * hkv) * d, device="cuda", dtype=torch.float16) * 0.3
    q = qkv[:, : hq * d].view(total, hq, d)
    k = qkv[:, hq * d : (hq + hkv) * d].view(total, hkv, d)
    v = qkv[:, (hq + hkv) * d :].view(total, hkv, d)
    lens = torch.randint(1, S + 1, (B,), dtype=torch.int32)
    lens[0], lens[1] = S, 1
    b_start = (torch.arange(B, dtype=torch.int32) * S).cuda()
    out = K().flash_attention2_no_pad(q, k, v, LOG2E / math.sqrt(d), b_start, lens.cuda(), S)
    ref = ops.varlen_causal_attention(q.cpu(), k.cpu(), v.cpu(), b_start.cpu(), lens, 1.0 / math.sqrt(d))
    valid = torch.zeros(total, dtype=torch.bool)
    for s0, n in zip(b_start.tolist(), lens.tolist()):
        valid[s0 : s0 + n] = True
    close(out.cpu()[valid], ref[valid], **ATT_TOL)


def test_flash_attention_nopad_first_token_sees_only_itself():
    d = 64
    q = torch.randn(40, 4, d, device="cuda", dtype=torch.float16)
    k = torch.randn(40, 4, d, device="cuda", dtype=torch.float16)
    v = torch.randn(40, 4, d, device="cuda", dtype=torch.float16)
    out = K().flash_attention2_no_pad(q, k, v, LOG2E / math.sqrt(d), torch.tensor([0, 25], dtype=torch.int32, device="cuda"),
                                      torch.tensor([25, 15], dtype=torch.int32, device="cuda"), 25)
    close(out[0], v[0], **ATT_TOL)
    close(out[25], v[25], **ATT_TOL)  # no leak from the previous sequence


# --------------------------------------------------------------------------- #
# dense linear (tcgen05)
# --------------------------------------------------------------------------- #
@pytest.mark.parametrize("m,n,k", [(1, 128, 64), (1, 256, 512), (8, 2048, 2048), (32, 4096, 4096), (33, 130, 384),
                                   (128, 768, 1024), (200, 1000, 320), (300, 512, 4096), (32, 512, 14336)])
@pytest.mark.parametrize("dtype", [torch.float16, torch.bfloat16])
def test_linear_matches_oracle(m, n, k, dtype):
    x = torch.randn(m, k, device="cuda", dtype=dtype) * 0.5
    w = torch.randn(n, k, device="cuda", dtype=dtype) * 0.05
    out = K().linear(x, w)
    ref = x.float().cpu() @ w.float().cpu().T
    tol = GEMM_TOL if dtype == torch.float16 else dict(rtol=1.6e-2, atol=1.6e-2)
    close(out, ref.to(dtype), **tol)


def test_linear_bias_leading_dims_and_determinism():
    x = torch.randn(2, 3, 4096, device="cuda", dtype=torch.float16) * 0.5
    w = torch.randn(1024, 4096, device="cuda", dtype=torch.float16) * 0.05
    b = torch.randn(1024, device="cuda", dtype=torch.float16)
    out = K().linear(x, w, b)
    assert out.shape == (2, 3, 1024)
    close(out, ops.linear(x.cpu(), w.cpu(), b.cpu()), **GEMM_TOL)
    # split-K reduction is ordered: bitwise reproducible
    for _ in range(3):
        assert torch.equal(K().linear(x, w, b), out)


def test_linear_llama3_lm_head_slice():
    x = torch.randn(32, 4096, device="cuda", dtype=torch.float16)
    w = torch.randn(16032, 4096, device="cuda", dtype=torch.float16) * 0.02
    out = K().linear(x, w)
    close(out, (x.float() @ w.float().T).half(), **GEMM_TOL)


# --------------------------------------------------------------------------- #
# quantised GEMMs
# --------------------------------------------------------------------------- #
def test_w4a16_golden():
    for c in load_golden("w4a16")["cases"]:
        g = to_cuda(c)
        out = K().w4a16_matmul(g["x"], g["qweight"], g["scales"], g["zeros"], group_size=c["group_size"], bias=g["bias"])
        close(out, c["out"], **GEMM_TOL)


@pytest.mark.parametrize("m,n,k", [(1, 256, 512), (8, 512, 1024), (32, 4096, 4096), (33, 130, 384), (100, 256, 2048),
                                   (32, 512, 14336)])
@pytest.mark.parametrize("gs", [32, 128])
def test_w4a16_matches_oracle(m, n, k, gs):
    x = torch.randn(m, k, device="cuda", dtype=torch.float16) * 0.5
    w = torch.randn(n, k, dtype=torch.float32) * 0.05
    qw, sc, zp = ops.quantize_int4_groupwise(w, gs)
    out = K().w4a16_matmul(x, qw.cuda(), sc.cuda(), zp.cuda(), group_size=gs)
    close(out, ops.w4a16_matmul(x.cpu(), qw, sc, zp, gs), **GEMM_TOL)


def test_w4a16_non_integer_zero_points_and_bias():
    m, n, k, gs = 5, 256, 512, 128
    x = torch.randn(m, k, device="cuda", dtype=torch.float16) * 0.5
    qw = torch.randint(-(2**31), 2**31 - 1, (n, k // 8), dtype=torch.int64).to(torch.int32)
    sc = torch.rand(n, k // gs) * 0.01 + 0.001
    zp = torch.rand(n, k // gs) * 15
    bias = torch.randn(n)
    out = K().w4a16_matmul(x, qw.cuda(), sc.cuda(), zp.cuda(), group_size=gs, bias=bias.cuda())
    close(out, ops.w4a16_matmul(x.cpu(), qw, sc, zp, gs, bias), **GEMM_TOL)


@pytest.mark.parametrize("m,n,k", [(32, 384, 4096), (7, 130, 1152)])
def test_w4a16_single_fractional_zero_point_switches_whole_tile(m, n, k):
    # integer zero points are folded into the operand exactly; one fractional entry anywhere in a tile's rows
    # must move that tile to the activation-row-sum correction without changing the result
    gs = 128
    x = torch.randn(m, k, device="cuda", dtype=torch.float16) * 0.5
    w = torch.randn(n, k, dtype=torch.float32) * 0.05
    qw, sc, zp = ops.quantize_int4_groupwise(w, gs)
    zp = zp.clone()
    zp[n // 2, -1] += 0.37
    zp[0, 0] = 1500.0          # integer but outside the foldable range
    out = K().w4a16_matmul(x, qw.cuda(), sc.cuda(), zp.cuda(), group_size=gs)
    close(out, ops.w4a16_matmul(x.cpu(), qw, sc, zp, gs), rtol=2e-3, atol=2e-3 + 2e-3 * float(sc.max()) * 1500)


def test_w4a16_unpack_order_is_bit_exact():
    # one-hot activations read single weights back: every (n, k) must land on nibble k%8 of word k//8
    n, k, gs = 128, 128, 128
    qw = torch.randint(-(2**31), 2**31 - 1, (n, k // 8), dtype=torch.int64).to(torch.int32)
    x = torch.eye(k, dtype=torch.float16, device="cuda")
    out = K().w4a16_matmul(x, qw.cuda(), torch.ones(n, 1, device="cuda"), torch.zeros(n, 1, device="cuda"), group_size=gs)
    assert torch.equal(out.cpu().T.to(torch.int64), ops.unpack_int4(qw))


# ---- kernel-native (load-time repacked) W4A16 layout: same product, bit for bit ----
def _w4_packed(qw, sc, zp, gs):
    return K().w4a16_pack(qw.cuda(), sc.cuda(), zp.cuda(), group_size=gs)


def test_w4a16_pack_matches_oracle():
    n, k, gs = 300, 1152, 128
    qw = torch.randint(-(2**31), 2**31 - 1, (n, k // 8), dtype=torch.int64).to(torch.int32)
    sc = torch.rand(n, k // gs) + 0.5
    zp = torch.randint(0, 16, (n, k // gs)).float()
    pk = _w4_packed(qw, sc, zp, gs)
    assert torch.equal(pk.qweight.cpu(), ops.pack_w4_qweight(qw))
    assert torch.equal(pk.scales.cpu(), ops.pack_w4_table(sc))
    assert torch.equal(pk.zeros.cpu(), ops.pack_w4_table(zp))
    assert pk.zeros_foldable
    zp[7, 2] = 3.5
    assert not _w4_packed(qw, sc, zp, gs).zeros_foldable


@pytest.mark.parametrize("m,n,k", [(1, 256, 512), (8, 512, 1024), (32, 4096, 4096), (33, 130, 384), (100, 256, 2048),
                                   (32, 512, 14336), (16, 640, 1792), (3, 130, 768), (32, 1000, 2304), (7, 128, 5120)])
@pytest.mark.parametrize("gs", [32, 128])
def test_w4a16_packed_matches_oracle_and_reference_layout(m, n, k, gs):
    x = torch.randn(m, k, device="cuda", dtype=torch.float16) * 0.5
    w = torch.randn(n, k, dtype=torch.float32) * 0.05
    qw, sc, zp = ops.quantize_int4_groupwise(w, gs)
    bias = torch.randn(n)
    out = K().w4a16_matmul_packed(x, _w4_packed(qw, sc, zp, gs), bias=bias.cuda())
    close(out, ops.w4a16_matmul(x.cpu(), qw, sc, zp, gs, bias), **GEMM_TOL)
    # same exact integer operand values, same accumulation order: identical to the reference-layout kernel
    assert torch.equal(out, K().w4a16_matmul(x, qw.cuda(), sc.cuda(), zp.cuda(), group_size=gs, bias=bias.cuda()))


def test_w4a16_packed_fractional_zero_points():
    m, n, k, gs = 9, 384, 2048, 256
    x = torch.randn(m, k, device="cuda", dtype=torch.float16) * 0.5
    qw = torch.randint(-(2**31), 2**31 - 1, (n, k // 8), dtype=torch.int64).to(torch.int32)
    sc = torch.rand(n, k // gs) * 0.01 + 0.001
    zp = torch.rand(n, k // gs) * 15
    pk = _w4_packed(qw, sc, zp, gs)
    assert not pk.zeros_foldable
    close(K().w4a16_matmul_packed(x, pk), ops.w4a16_matmul(x.cpu(), qw, sc, zp, gs), **GEMM_TOL)


def test_w4a16_packed_unpack_order_is_bit_exact():
    n, k, gs = 128, 256, 128
    qw = torch.randint(-(2**31), 2**31 - 1, (n, k // 8), dtype=torch.int64).to(torch.int32)
    x = torch.eye(k, dtype=torch.float16, device="cuda")
    pk = _w4_packed(qw, torch.ones(n, k // gs), torch.zeros(n, k // gs), gs)
    out = K().w4a16_matmul_packed(x, pk)
    assert torch.equal(out.cpu().T.to(torch.int64), ops.unpack_int4(qw))


@pytest.mark.parametrize("n,k", [(6144, 4096), (4096, 4096), (28672, 4096), (4096, 14336)])
@pytest.mark.parametrize("m", [1, 32])
def test_w4a16_packed_llama3_8b_projection_shapes(m, n, k):
    gs = 128
    torch.manual_seed(1)
    x = torch.randn(m, k, device="cuda", dtype=torch.float16) * 0.5
    qw = torch.randint(-(2**31), 2**31 - 1, (n, k // 8), device="cuda", dtype=torch.int64).to(torch.int32)
    sc = torch.rand(n, k // gs, device="cuda") * 0.004 + 0.001
    zp = torch.randint(0, 16, (n, k // gs), device="cuda").float()
    out = K().w4a16_matmul_packed(x, K().w4a16_pack(qw, sc, zp, group_size=gs))
    assert torch.equal(out, K().w4a16_matmul(x, qw, sc, zp, group_size=gs))
    for _ in range(2):
        assert torch.equal(out, K().w4a16_matmul_packed(x, K().w4a16_pack(qw, sc, zp, group_size=gs)))


def test_w8a16_golden():
    for c in load_golden("w8a16")["cases"]:
        x = c["x"].cuda()
        for key in ("fp8_block", "int8_channel", "fp8_channel"):
            d = c[key]
            out = K().w8a16_matmul(x, d["qweight"].cuda(), d["scales"].cuda(), group_n=d["group_n"], group_k=d["group_k"])
            close(out, d["out"], **GEMM_TOL)


@pytest.mark.parametrize("m,n,k", [(1, 512, 256), (8, 2048, 2048), (128, 768, 1024), (33, 130, 384)])
def test_w8a16_matches_oracle(m, n, k):
    x = torch.randn(m, k, device="cuda", dtype=torch.float16) * 0.5
    w = torch.randn(n, k) * 0.05
    qw = w.to(torch.float8_e4m3fn).view(torch.uint8)
    sc = torch.rand((n + 127) // 128, (k + 127) // 128) + 0.5
    out = K().w8a16_matmul(x, qw.cuda(), sc.cuda(), group_n=128, group_k=128)
    close(out, ops.w8a16_matmul(x.cpu(), qw, sc, 128, 128), **GEMM_TOL)
    qi, si = ops.quantize_int8_per_channel(w)
    out = K().w8a16_matmul(x, qi.cuda(), si.cuda(), group_n=1, group_k=k)
    close(out, ops.w8a16_matmul(x.cpu(), qi, si, 1, k), **GEMM_TOL)


def test_fp8_dequant_is_exact_for_every_code():
    # each finite e4m3 code, read back through a one-hot activation, must equal its exact value
    codes = torch.arange(256, dtype=torch.int32).to(torch.uint8)
    finite = (codes & 0x7F) != 0x7F
    safe = torch.where(finite, codes, torch.zeros_like(codes))   # NaN codes would poison every dot product
    qw = safe.repeat(128, 1).contiguous()                        # [128, 256]
    x = torch.eye(256, dtype=torch.float16, device="cuda")
    out = K().w8a16_matmul(x, qw.cuda(), torch.ones(1, 1, device="cuda"), group_n=128, group_k=256)
    expect = codes.view(torch.float8_e4m3fn).float()
    assert torch.equal(out.cpu()[:, 0].float()[finite], expect[finite])
    assert torch.equal(out.cpu()[:, 77].float()[finite], expect[finite])


def test_smoothquant_golden_and_quantiser_codes():
    for c in load_golden("w8a8")["cases"]:
        g = to_cuda(c)
        out = K().smoothquant_matmul(g["x"], g["qweight"], g["weight_scales"], bias=g["bias"])
        # the golden was recorded on the CPU; an activation code may differ by one count at a truncation
        # boundary: |delta| <= max|w_dequant| * a_scale ~ 3e-3 here
        close(out, c["out"], rtol=2e-3, atol=4e-3)
    from lite_llama_b200.kernels.quantization.w8a8 import quantize_activations_int8

    x = torch.randn(64, 2048, device="cuda", dtype=torch.float16) * 0.5
    q, s = quantize_activations_int8(x)
    q_ref, s_ref = ops.quantize_activations_int8(x.cpu())
    torch.testing.assert_close(s.cpu(), s_ref, rtol=1e-6, atol=0)
    # codes may differ by one only at exact integers
    diff = (q.cpu().int() - q_ref.int()).abs()
    assert diff.max() <= 1 and (diff != 0).float().mean() < 1e-3


@pytest.mark.parametrize("m,n,k", [(1, 256, 512), (8, 512, 1024), (64, 2048, 2048), (256, 3584, 3584), (33, 130, 384)])
def test_smoothquant_matches_oracle(m, n, k):
    x = torch.randn(m, k, device="cuda", dtype=torch.float16) * 0.5
    w = torch.randn(n, k) * 0.05
    scale = w.abs().amax(-1) / 127.0
    qw = (w / scale.unsqueeze(-1)).round().clamp(-127, 127).to(torch.int8)
    out = K().smoothquant_matmul(x, qw.cuda(), scale.cuda())
    # compare on the kernel's own activation codes (they may differ from IEEE by one count at ties)
    from lite_llama_b200.kernels.quantization.w8a8 import quantize_activations_int8

    qa, sa = quantize_activations_int8(x)
    acc = qa.cpu().to(torch.int64) @ qw.to(torch.int64).T
    ref = (acc.float() * sa.cpu().unsqueeze(-1) * scale.unsqueeze(0)).half()
    close(out, ref, rtol=1e-3, atol=5e-4)
    close(out, ops.smoothquant_matmul(x.cpu(), qw, scale), rtol=2e-2, atol=2e-2)


# --------------------------------------------------------------------------- #
# MoE: align (bit-exact), router, grouped GEMMs
# --------------------------------------------------------------------------- #
def test_moe_align_golden_bit_exact():
    for c in load_golden("moe_align")["cases"]:
        s, e, n = K().moe_align_block_size(c["topk_ids"].cuda(), c["block_size"], c["num_experts"])
        assert torch.equal(s.cpu(), c["sorted_ids"]) and torch.equal(e.cpu(), c["expert_ids"]) and torch.equal(n.cpu(), c["num_post"])


@pytest.mark.parametrize("tokens,experts,top_k,block", [(1, 8, 2, 16), (37, 128, 8, 32), (513, 128, 8, 64), (4096, 60, 4, 64),
                                                        (3, 1, 1, 16)])
@pytest.mark.parametrize("dt", [torch.int32, torch.int64])
def test_moe_align_matches_oracle_bit_exact(tokens, experts, top_k, block, dt):
    ids = torch.randint(0, experts, (tokens, top_k), dtype=dt)
    s, e, n = K().moe_align_block_size(ids.cuda(), block, experts)
    s_ref, e_ref, n_ref = ops.moe_align_block_size(ids, block, experts)
    assert torch.equal(n.cpu(), n_ref) and torch.equal(s.cpu(), s_ref) and torch.equal(e.cpu(), e_ref)


@pytest.mark.parametrize("tokens,experts,top_k", [(1, 128, 8), (37, 128, 8), (5, 8, 2), (64, 60, 4), (3, 512, 8)])
def test_moe_route_topk_matches_oracle(tokens, experts, top_k):
    logits = (torch.randn(tokens, experts) * 2).half()
    w, ids = K().route_topk(logits.cuda(), top_k, True)
    probs = torch.softmax(logits.float(), dim=-1)
    w_ref, ids_ref = torch.topk(probs, top_k, dim=-1)
    w_ref = (w_ref / w_ref.sum(-1, keepdim=True)).half()
    # ids must agree wherever the k-th and (k+1)-th probabilities are distinguishable
    srt = probs.sort(dim=-1, descending=True).values
    decidable = ((srt[:, :top_k] - srt[:, 1 : top_k + 1]) > 1e-6).all(dim=-1) if experts > top_k else torch.ones(tokens, dtype=torch.bool)
    assert torch.equal(ids.cpu()[decidable], ids_ref[decidable])
    close(w.cpu()[decidable], w_ref[decidable], rtol=2e-3, atol=1e-4)


def test_fused_moe_golden():
    for c in load_golden("fused_moe")["cases"]:
        g = to_cuda(c)
        out = K().fused_moe(g["hidden"], g["w1"], g["w2"], g["topk_weights"], g["topk_ids"],
                            w1_scale=g.get("w1_scale"), w2_scale=g.get("w2_scale"),
                            group_n=c.get("group_n", 0), group_k=c.get("group_k", 0))
        close(out, c["out"], rtol=5e-3, atol=2e-4)


@pytest.mark.parametrize("num_tokens", [1, 3, 37, 128])
@pytest.mark.parametrize("num_experts,top_k", [(8, 2), (128, 8)])
def test_fused_moe_matches_oracle(num_tokens, num_experts, top_k):
    hidden, inter = 256, 128
    x = (torch.randn(num_tokens, hidden) / hidden**0.5).half()
    w1 = (torch.randn(num_experts, 2 * inter, hidden) / hidden**0.5).half()
    w2 = (torch.randn(num_experts, hidden, inter) / inter**0.5).half()
    ids = torch.randint(0, num_experts, (num_tokens, top_k))
    tw = torch.softmax(torch.randn(num_tokens, top_k), dim=-1).half()
    out = K().fused_moe(x.cuda(), w1.cuda(), w2.cuda(), tw.cuda(), ids.cuda())
    ref = ops.fused_moe(x, w1, w2, tw, ids)
    close(out, ref, rtol=5e-3, atol=5e-4)


@pytest.mark.parametrize("kind", ["fp8", "int8"])
def test_fused_moe_quantised_experts_qwen3_shape(kind):
    # Qwen3-30B-A3B slice: hidden 2048, moe_intermediate 768, 128x128 fp8 blocks (config 5), fewer experts
    tokens, E, top_k, hidden, inter = 32, 16, 4, 2048, 768
    x = (torch.randn(tokens, hidden) / hidden**0.5).half()
    w1f = torch.randn(E, 2 * inter, hidden) / hidden**0.5
    w2f = torch.randn(E, hidden, inter) / inter**0.5
    if kind == "fp8":
        w1, w2 = w1f.to(torch.float8_e4m3fn).view(torch.uint8), w2f.to(torch.float8_e4m3fn).view(torch.uint8)
        s1 = torch.rand(E, 2 * inter // 128, hidden // 128) + 0.5
        s2 = torch.rand(E, hidden // 128, inter // 128) + 0.5
        gn = gk = 128
    else:
        w1, s1 = ops.quantize_int8_per_channel(w1f)
        w2, s2 = ops.quantize_int8_per_channel(w2f)
        gn, gk = 1, 1 << 30
    ids = torch.randint(0, E, (tokens, top_k))
    tw = torch.softmax(torch.randn(tokens, top_k), dim=-1).half()
    out = K().fused_moe(x.cuda(), w1.cuda(), w2.cuda(), tw.cuda(), ids.cuda(), w1_scale=s1.cuda(), w2_scale=s2.cuda(),
                        group_n=gn, group_k=gk)
    ref = ops.fused_moe(x, w1, w2, tw, ids, s1, s2, gn, min(gk, 1 << 20))
    close(out, ref, rtol=5e-3, atol=1e-3)


@pytest.mark.parametrize("tp,g", [(4, 64), (8, 32)])
def test_fused_moe_sub_block_tensor_parallel_shard(tp, g):
    """One rank's expert shard of Qwen3-30B-A3B at TP = 4 / 8: 768 / tp intermediate columns per expert, which cuts the
    checkpoint's 128 x 128 scale blocks; scales refined to g = gcd(128, 768 / tp) and passed as group_n = group_k = g
    (the reference refuses these shards, lite_llama/models/linear.py:164-177)."""
    from lite_llama_b200.quantization.params import quantize_fp8_blockwise, reblock_scales

    tokens, E, top_k, hidden, inter = 32, 16, 4, 2048, 768
    il = inter // tp
    x = (torch.randn(tokens, hidden) / hidden**0.5).half()
    gate = torch.randn(E, inter, hidden) / hidden**0.5
    up = torch.randn(E, inter, hidden) / hidden**0.5
    down = torch.randn(E, hidden, inter) / inter**0.5
    rank = 1
    lo, hi = rank * il, (rank + 1) * il
    parts = []
    for t in (gate, up, down):
        q, sc = quantize_fp8_blockwise(t)
        parts.append((q, reblock_scales(reblock_scales(sc, 128, g, 1), 128, g, 2)))
    (qg, sg), (qu, su), (qd, sd) = parts
    w1 = torch.cat([qg[:, lo:hi], qu[:, lo:hi]], dim=1).contiguous()
    s1 = torch.cat([sg[:, lo // g:hi // g], su[:, lo // g:hi // g]], dim=1).contiguous()
    w2 = qd[:, :, lo:hi].contiguous()
    s2 = sd[:, :, lo // g:hi // g].contiguous()
    ids = torch.randint(0, E, (tokens, top_k))
    tw = torch.softmax(torch.randn(tokens, top_k), dim=-1).half()
    out = K().fused_moe(x.cuda(), w1.cuda(), w2.cuda(), tw.cuda(), ids.cuda(), w1_scale=s1.cuda(), w2_scale=s2.cuda(),
                        group_n=g, group_k=g)
    ref = ops.fused_moe(x, w1, w2, tw, ids, s1, s2, g, g)
    close(out, ref, rtol=5e-3, atol=1e-3)


def test_fused_moe_zero_routing_weight_drops_the_slot():
    hidden, inter, E, top_k = 128, 64, 4, 2
    x = torch.randn(5, hidden).half()
    w1 = (torch.randn(E, 2 * inter, hidden) / hidden**0.5).half()
    w2 = (torch.randn(E, hidden, inter) / inter**0.5).half()
    ids = torch.randint(0, E, (5, top_k))
    tw = torch.rand(5, top_k).half()
    tw[:, 1] = 0
    out = K().fused_moe(x.cuda(), w1.cuda(), w2.cuda(), tw.cuda(), ids.cuda())
    close(out, ops.fused_moe(x, w1, w2, tw, ids), rtol=5e-3, atol=2e-3)


# --------------------------------------------------------------------------- #
# programmatic dependent launch: overlapped kernel chains must be bit-identical to serialised ones
# --------------------------------------------------------------------------- #
def test_pdl_kernel_chain_llama_shapes_bit_identical():
    """One Llama-3-8B MLP block at batch 32 (rmsnorm -> gate|up W4A16 -> swiglu -> down W4A16), 12 rounds feeding
    each round's output back in, with the launch attribute off and on. The GEMMs prefetch weights and scale tables
    before griddepcontrol.wait; activations, outputs and the split-K workspace must only be touched after it."""
    from lite_llama_b200 import _lib

    lib = _lib.load()
    torch.manual_seed(0)
    h, inter, m = 4096, 14336, 32
    dev = "cuda"
    qgu = torch.randint(-(2**31), 2**31 - 1, (2 * inter, h // 8), device=dev, dtype=torch.int64).to(torch.int32)
    sgu = torch.rand(2 * inter, h // 128, device=dev) * 0.004
    zgu = torch.randint(0, 16, (2 * inter, h // 128), device=dev).float()
    qd = torch.randint(-(2**31), 2**31 - 1, (h, inter // 8), device=dev, dtype=torch.int64).to(torch.int32)
    sd = torch.rand(h, inter // 128, device=dev) * 0.004
    zd = torch.randint(0, 16, (h, inter // 128), device=dev).float()
    wn = torch.ones(h, device=dev, dtype=torch.float16)
    x0 = torch.randn(m, 1, h, device=dev, dtype=torch.float16)

    def run(pdl):
        old = lib.b2l_set_pdl(pdl)
        try:
            x = x0.clone()
            res = torch.zeros_like(x0)
            for _ in range(12):
                y, res = K().skip_rmsnorm(x, res, wn, 1e-5)
                gu = K().w4a16_matmul(y.view(m, h), qgu, sgu, zgu, group_size=128)
                act = K().swiglu_forward(gu[:, :inter], gu[:, inter:])
                x = K().w4a16_matmul(act, qd, sd, zd, group_size=128).view(m, 1, h)
            torch.cuda.synchronize()
            return x.cpu(), res.cpu()
        finally:
            lib.b2l_set_pdl(old)

    a = run(0)
    b = run(1)
    c = run(1)
    assert torch.isfinite(a[0].float()).all()
    assert torch.equal(a[0], b[0]) and torch.equal(a[1], b[1])
    assert torch.equal(b[0], c[0])


# --------------------------------------------------------------------------- #
# stream-K schedule of the quantised GEMMs (csrc/gemm_quant.cu): CTA ranges that start and end inside tiles
# --------------------------------------------------------------------------- #
def _plan(kind, m, n, k, gk):
    import ctypes

    from lite_llama_b200 import _lib

    out = (ctypes.c_int * 10)()
    _lib.check(_lib.load().b2l_quant_gemm_plan(kind, m, n, k, gk, out, None))
    return list(out)


@pytest.mark.parametrize("m,n,k", [(16, 640, 1792), (3, 130, 768), (32, 1000, 2304), (64, 384, 4096), (7, 128, 5120)])
def test_w4a16_stream_k_piece_boundaries(m, n, k):
    # tile counts and K depths chosen so that CTA ranges cut tiles at odd places, several CTAs share a tile and one
    # CTA spans up to three tiles; N not a multiple of 128 puts rows past N into the last tile
    gs = 128
    assert _plan(0, m, n, k, gs)[0] > 0, "shape is expected to take the stream-K schedule"
    x = torch.randn(m, k, device="cuda", dtype=torch.float16) * 0.5
    w = torch.randn(n, k, dtype=torch.float32) * 0.05
    qw, sc, zp = ops.quantize_int4_groupwise(w, gs)
    bias = torch.randn(n)
    args = (x, qw.cuda(), sc.cuda(), zp.cuda())
    out = K().w4a16_matmul(*args, group_size=gs, bias=bias.cuda())
    close(out, ops.w4a16_matmul(x.cpu(), qw, sc, zp, gs, bias), **GEMM_TOL)
    for _ in range(3):   # partial sums are combined in CTA order, whoever finishes last: bit-stable
        assert torch.equal(out, K().w4a16_matmul(*args, group_size=gs, bias=bias.cuda()))


def test_w4a16_stream_k_group_256_and_fractional_zero_points():
    m, n, k, gs = 9, 384, 2048, 256
    assert _plan(0, m, n, k, gs)[0] > 0
    x = torch.randn(m, k, device="cuda", dtype=torch.float16) * 0.5
    qw = torch.randint(-(2**31), 2**31 - 1, (n, k // 8), dtype=torch.int64).to(torch.int32)
    sc = torch.rand(n, k // gs) * 0.01 + 0.001
    zp = torch.randint(0, 16, (n, k // gs)).float()
    out = K().w4a16_matmul(x, qw.cuda(), sc.cuda(), zp.cuda(), group_size=gs)
    close(out, ops.w4a16_matmul(x.cpu(), qw, sc, zp, gs), **GEMM_TOL)
    zp[200, 3] += 0.25      # one fractional zero point: the CTAs that hold it switch to the row-sum correction
    out = K().w4a16_matmul(x, qw.cuda(), sc.cuda(), zp.cuda(), group_size=gs)
    close(out, ops.w4a16_matmul(x.cpu(), qw, sc, zp, gs), **GEMM_TOL)


@pytest.mark.parametrize("m,n,k", [(5, 640, 1152), (32, 2048, 2048), (64, 300, 896)])
def test_w8a16_stream_k_block_scales(m, n, k):
    assert _plan(1, m, n, k, 128)[0] > 0
    x = torch.randn(m, k, device="cuda", dtype=torch.float16) * 0.5
    w = torch.randn(n, k) * 0.05
    qw = w.to(torch.float8_e4m3fn).view(torch.uint8)
    sc = torch.rand((n + 127) // 128, (k + 127) // 128) + 0.5
    bias = torch.randn(n, dtype=torch.float16)
    out = K().w8a16_matmul(x, qw.cuda(), sc.cuda(), group_n=128, group_k=128, bias=bias.cuda())
    close(out, ops.w8a16_matmul(x.cpu(), qw, sc, 128, 128, bias), **GEMM_TOL)
    qi = torch.randint(-127, 128, (n, k), dtype=torch.int8)
    si = torch.rand((n + 63) // 64, (k + 127) // 128) * 0.01
    out = K().w8a16_matmul(x, qi.cuda(), si.cuda(), group_n=64, group_k=128)
    close(out, ops.w8a16_matmul(x.cpu(), qi, si, 64, 128), **GEMM_TOL)


@pytest.mark.parametrize("n,k", [(6144, 4096), (4096, 4096), (28672, 4096), (4096, 14336)])
@pytest.mark.parametrize("m", [1, 32])
def test_w4a16_llama3_8b_projection_shapes(m, n, k):
    # full BASELINE shapes: compared on the GPU with an fp32 matmul over the dequantised weights (same formula as
    # oracle/ops.py:w4a16_matmul, which takes minutes at this size on the CPU)
    gs = 128
    torch.manual_seed(1)
    x = torch.randn(m, k, device="cuda", dtype=torch.float16) * 0.5
    qw = torch.randint(-(2**31), 2**31 - 1, (n, k // 8), device="cuda", dtype=torch.int64).to(torch.int32)
    sc = torch.rand(n, k // gs, device="cuda") * 0.004 + 0.001
    zp = torch.randint(0, 16, (n, k // gs), device="cuda").float()
    out = K().w4a16_matmul(x, qw, sc, zp, group_size=gs)
    shifts = torch.arange(8, device="cuda", dtype=torch.int32) * 4
    nib = ((qw.unsqueeze(-1) >> shifts) & 0xF).reshape(n, k).float()
    wd = (nib - zp.repeat_interleave(gs, dim=1)) * sc.repeat_interleave(gs, dim=1)
    ref = x.float() @ wd.T
    torch.testing.assert_close(out.float(), ref, rtol=2e-3, atol=2e-3 * float(ref.abs().max()))


# --------------------------------------------------------------------------- #
# batch-1 Llama-3-8B geometry, op by op (the decode step that stalled lives at these shapes)
# --------------------------------------------------------------------------- #
def test_bs1_llama_geometry_every_op_of_the_layer():
    torch.manual_seed(0)
    h, hq, hkv, d, inter, V = 4096, 32, 8, 128, 14336, 128256
    dev = "cuda"
    # skip_rmsnorm: one row of 4096
    x = torch.randn(1, 1, h, device=dev, dtype=torch.float16)
    res = torch.randn(1, 1, h, device=dev, dtype=torch.float16)
    w = torch.randn(h, device=dev, dtype=torch.float16) * 0.1 + 1
    y, r = K().skip_rmsnorm(x, res.clone(), w, 1e-5)
    yr, rr = ops.skip_rmsnorm(x.cpu(), res.cpu(), w.cpu(), 1e-5)
    close(y.cpu(), yr, rtol=2e-3, atol=2e-3)
    close(r.cpu(), rr, rtol=1e-3, atol=1e-3)
    # fused qkv projection at M = 1 (W4A16), rope + cache write of the single token, decode attention over a
    # 200-token history in the fused pool with the 256 bucket, o projection
    wq = torch.randn((hq + 2 * hkv) * d, h) * 0.02
    qw, sc, zp = ops.quantize_int4_groupwise(wq, 128)
    xin = y.view(1, h)
    qkv = K().w4a16_matmul_packed(xin, K().w4a16_pack(qw.to(dev), sc.to(dev), zp.to(dev), group_size=128))
    close(qkv.cpu(), ops.w4a16_matmul(xin.cpu(), qw, sc, zp, 128), rtol=2e-3, atol=2e-3)
    ctx = 200
    pool = torch.randn(512, 2 * hkv, d, device=dev, dtype=torch.float16) * 0.5
    table = torch.randperm(512, device=dev)[:256].to(torch.int32).view(1, 256)
    cos = torch.randn(1, 1, d, device=dev, dtype=torch.float16)
    sin = torch.randn(1, 1, d, device=dev, dtype=torch.float16)
    q3 = qkv[:, : hq * d].view(1, hq, d)
    k3 = qkv[:, hq * d:(hq + hkv) * d].view(1, hkv, d)
    v3 = qkv[:, (hq + hkv) * d:].view(1, hkv, d)
    row = table[:, ctx - 1].clone()
    ref_q = ops.rope_half_split(q3.cpu().clone(), cos.cpu(), sin.cpu(), 1, 1)
    ref_k = ops.rope_half_split(k3.cpu().clone(), cos.cpu(), sin.cpu(), 1, 1)
    v_before = v3.clone()
    K().rope_kv_write(q3, k3, v3, cos, sin, row, pool, 1, 1)
    close(q3.cpu(), ref_q, rtol=2e-3, atol=2e-3)
    assert torch.equal(pool[row.long(), :hkv], k3) and torch.equal(pool[row.long(), hkv:], v_before)
    close(k3.cpu(), ref_k, rtol=2e-3, atol=2e-3)
    seq = torch.tensor([ctx], dtype=torch.int32, device=dev)
    req = torch.zeros(1, dtype=torch.int32, device=dev)
    att = K().flash_decoding(q3, pool[:, :hkv], pool[:, hkv:], 1 / math.sqrt(d), table, req, seq, 256)
    ref = ops.paged_decode_attention(q3.cpu(), pool[:, :hkv].cpu(), pool[:, hkv:].cpu(), table.cpu(), req.cpu(), seq.cpu(),
                                     1 / math.sqrt(d))
    close(att.cpu(), ref, **ATT_TOL)
    # gate|up with the swiglu epilogue and down at M = 1
    wgu = torch.randn(2 * inter, h) * 0.02
    qg, sg, zg = (t.to(dev) for t in ops.quantize_int4_groupwise(wgu, 128))
    from lite_llama_b200.kernels.quantization import interleave_gate_up

    act = K().w4a16_matmul_packed(xin, K().w4a16_pack(interleave_gate_up(qg), interleave_gate_up(sg), interleave_gate_up(zg),
                                                      group_size=128), swiglu=True)
    gu = K().w4a16_matmul(xin, qg, sg, zg, group_size=128)
    # same arithmetic; interleaving moves rows to other tiles, so stream-K cuts their K range at other raw blocks and
    # the fp32 partial sums are grouped differently: equal up to the last fp16 bit, not bit for bit (the bit-exact
    # comparison on unshared tiles is test_w4a16_swiglu_epilogue_is_bit_identical_to_gemm_then_swiglu)
    close(act.cpu(), K().swiglu_forward(gu[:, :inter], gu[:, inter:]).cpu(), rtol=2e-3, atol=1e-4)
    # lm_head: the full 128256 x 4096 fp16 matrix at M = 1
    lm = torch.randn(V, h, device=dev, dtype=torch.float16) * 0.02
    logits = K().linear(xin, lm)
    close(logits.cpu(), (xin.float().cpu() @ lm.float().cpu().T), rtol=2e-3, atol=2e-3)


def test_argmax_rows_matches_torch_and_breaks_ties_low():
    for rows, n, dtype in [(32, 128256, torch.float16), (1, 151936, torch.float16), (3, 1000, torch.bfloat16), (5, 7, torch.float16)]:
        x = torch.randn(rows, n, device="cuda", dtype=dtype)
        assert torch.equal(K().argmax_rows(x), x.float().argmax(-1))
        view = torch.randn(rows, 2, n, device="cuda", dtype=dtype)[:, -1, :]      # strided rows, like logits[:, -1, :]
        assert torch.equal(K().argmax_rows(view), view.float().argmax(-1))
    t = torch.zeros(2, 4096, device="cuda", dtype=torch.float16)
    t[0, 100] = t[0, 3000] = 5.0
    t[1, 4095] = 1.0
    assert K().argmax_rows(t).tolist() == [100, 4095]


@pytest.mark.parametrize("m", [32, 36, 1])
@pytest.mark.parametrize("n,k", [(4096, 4096), (6144, 4096), (4096, 14336), (3072, 4096), (4096, 2048), (4096, 7168),
                                 (14336, 4096)])
def test_w4a16_streamk_back_to_back_launches_are_isolated(m, n, k):
    """Stream-K tiles are handed over through a persistent workspace with flag-in-data words that every launch must
    leave clean (csrc/gemm_quant.cu).  Same-shaped launches reuse the very same words: run a chain of launches over
    DIFFERENT weights without synchronising (PDL overlaps them) and require every result to be bit-identical to the
    one the same call gives in isolation -- a launch that picked up a predecessor's partial sums (stale cache line,
    word not cleared) would differ by whole tiles."""
    torch.manual_seed(7)
    g = 128
    x = (torch.randn(m, k, device="cuda", dtype=torch.float16) * 0.5)
    packed = []
    for i in range(6):
        qw = torch.randint(-(2**31), 2**31 - 1, (n, k // 8), device="cuda", dtype=torch.int64).to(torch.int32)
        sc = torch.rand(n, k // g, device="cuda") * 0.01 + 0.001
        zp = torch.randint(0, 16, (n, k // g), device="cuda").float()
        packed.append(K().w4a16_pack(qw, sc, zp, group_size=g))
    alone = []
    for pk in packed:
        torch.cuda.synchronize()
        torch.zeros(1 << 22, device="cuda").add_(1.0)          # another kernel in between
        torch.cuda.synchronize()
        alone.append(K().w4a16_matmul_packed(x, pk).clone())
    torch.cuda.synchronize()
    for rep in range(int(os.environ.get("B2L_TEST_REPS", "20"))):
        outs = [K().w4a16_matmul_packed(x, pk) for pk in packed]   # back to back, no synchronisation
        torch.cuda.synchronize()
        for i, (a, b) in enumerate(zip(alone, outs)):
            assert torch.equal(a, b), f"repetition {rep}, launch {i}: result differs from the isolated call"


@pytest.mark.parametrize("rows,n", [(1, 3584), (32, 4096), (256, 3584), (7, 896), (3, 128), (5, 8192)])
@pytest.mark.parametrize("with_residual", [True, False])
def test_skip_rmsnorm_quant_int8_is_the_two_ops_in_one_launch(rows, n, with_residual):
    """SmoothQuant decoder: norm + per-token int8 quantisation fused (csrc/elementwise.cu). q, scales and the updated
    residual must be bit-identical to skip_rmsnorm followed by quantize_activations_int8 (reference:
    skip_rmsnorm.py:192-234, quantization/w8a8.py:35-68); the oracle pins the pair end to end."""
    torch.manual_seed(rows * 131 + n)
    x = torch.randn(rows, n, device="cuda", dtype=torch.float16)
    res = torch.randn(rows, n, device="cuda", dtype=torch.float16) if with_residual else None
    w = (torch.randn(n, device="cuda", dtype=torch.float16) * 0.1 + 1.0)
    r1 = res.clone() if with_residual else None
    y, r1o = K().skip_rmsnorm(x, r1, w, 1e-6)
    q_ref, s_ref = K().quantize_activations_int8(y)
    r2 = res.clone() if with_residual else None
    q, s, r2o = K().skip_rmsnorm_quant_int8(x, r2, w, 1e-6)
    assert torch.equal(q, q_ref) and torch.equal(s, s_ref)
    assert torch.equal(r1o, r2o)
    # against the CPU restatement of both ops
    y_cpu, _ = ops.skip_rmsnorm(x.cpu(), res.cpu() if with_residual else None, w.cpu(), 1e-6)
    q_cpu, s_cpu = ops.quantize_activations_int8(y_cpu)
    torch.testing.assert_close(s.cpu(), s_cpu.float().view(-1), rtol=2e-3, atol=1e-6)
    assert int((q.cpu().int() - q_cpu.int()).abs().max()) <= 1     # a 1-ulp difference of the fp16 norm output moves a step


def test_smoothquant_prequant_gemm_is_the_second_half_of_smoothquant_matmul():
    torch.manual_seed(3)
    m, n, k = 48, 512, 896
    x = torch.randn(m, k, device="cuda", dtype=torch.float16)
    wq = torch.randint(-127, 128, (n, k), device="cuda", dtype=torch.int8)
    ws = torch.rand(n, device="cuda") * 0.01
    bias = torch.randn(n, device="cuda")
    full = K().smoothquant_matmul(x, wq, ws, bias=bias)
    qa, sa = K().quantize_activations_int8(x)
    half = K().smoothquant_matmul_prequant(qa, sa, wq, ws, bias=bias, out_dtype=torch.float16)
    assert torch.equal(full, half)
