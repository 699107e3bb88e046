"""Host side of the Torutar design: configuration parser, registry, weight mapping, cache and state shapes, row release
with kept first tokens, and the restatement's own invariants.  No GPU."""

from __future__ import annotations

import numpy as np
import pytest
import torch

import torutar_oracle as O
from lite_llama_b200.executor.layered_decoder import (aligned_columns, map_torutar_weights, parse_torutar_config,
                                                      random_torutar_tensors, torutar_tensor_shapes)
from lite_llama_b200.executor.model_config import LatentAttentionSpec, MlstmSpec, MoeMlpSpec, WindowAttentionSpec
from lite_llama_b200.executor.registry import lookup
from lite_llama_b200.executor.state_manager import RecurrentStateManager


def _config():
    return O.make_config([O.attention_layer(heads=6, kv_heads=2, dim=8, vdim=5, size=11, keep_first=3, rot=6, base=777.0, scale=0.3),
                          O.mlstm_layer(3, 4, 7, 9.5, mlp=None),
                          O.latent_layer(mlp=O.moe_mlp(4, 3, 5, 0.5, 1.3, 0)),
                          O.attention_layer(heads=6, kv_heads=2, dim=8, vdim=5, size=0, rot=6, base=777.0, kv_from=0, mlp=None)],
                         width=20, vocab=33, eps=1e-4, streams=3, taps=5, logit_scale=0.25)


def test_every_size_and_constant_comes_from_the_configuration():
    cfg = lookup("torutar").parse_config(_config())
    cfg.validate()
    assert (cfg.hidden_size, cfg.vocab_size, cfg.streams, cfg.input_conv, cfg.logit_scale, cfg.rms_norm_eps, cfg.max_seq_len) == \
        (20, 33, 3, 5, 0.25, 1e-4, 0)
    assert cfg.embed_norm and cfg.sublayer_gate and cfg.norm_weight_offset == 0.0
    a, m, l, b = (x.mixer for x in cfg.layers)
    assert isinstance(a, WindowAttentionSpec) and (a.heads, a.kv_heads, a.head_dim, a.v_head_dim) == (6, 2, 8, 5)
    assert (a.window, a.keep_first, a.rot_dims, a.rot_base, a.scale, a.pairing, a.kv_from) == (11, 3, 6, 777.0, 0.3, "halves", None)
    assert isinstance(m, MlstmSpec) and m.gate_cap == 9.5 and m.state_shape == (3, 36)          # 28 + 4 + 1, padded to 16 bytes
    assert isinstance(l, LatentAttentionSpec) and l.element_gate and l.pairing == "neighbours" and l.window == 0
    assert (l.q_rank, l.kv_rank, l.rot_dim, l.rot_dims, l.rot_base) == (7, 6, 4, 4, 500.0)
    assert b.kv_from == 0 and b.window == 0 and b.keep_first == 0
    assert cfg.attention_layers() == [0, 2] and cfg.cache_readers() == [0, 2, 3] and cfg.recurrent_layers() == [1]
    f = cfg.layers[0].mlp
    assert isinstance(f, MoeMlpSpec) and (f.experts, f.top, f.ff, f.limit, f.scale) == (5, 2, 6, 0.9, 1.7)
    assert (f.shared_ff, f.shared_limit, f.scores, f.activation, f.renormalize, f.alpha) == (7, 0.6, "softmax", "clamped", True, 1.702)
    assert cfg.layers[2].mlp.shared_ff == 0 and cfg.layers[1].mlp is None


@pytest.mark.parametrize("break_it", [lambda c: c["layers"][0].update(type="lstm"), lambda c: c["layers"][0]["mlp"].update(kind="maxout"),
                                      lambda c: c["layers"][0]["mixer"].update(kv_heads=4), lambda c: c["layers"][3]["mixer"].update(kv_from=3),
                                      lambda c: c["layers"][3]["mixer"].update(kv_from=2), lambda c: c["layers"][3]["mixer"].update(dim=4, rot=None),
                                      lambda c: c["layers"][0]["mlp"]["router"].update(top=6)])
def test_what_does_not_fit_is_refused(break_it):
    raw = _config()
    break_it(raw)
    with pytest.raises(ValueError):
        parse_torutar_config(raw).validate()


def test_names_shapes_and_layouts_of_the_weights():
    raw = _config()
    cfg = parse_torutar_config(raw)
    assert torutar_tensor_shapes(cfg) == O.tensor_shapes(raw)
    t = random_torutar_tensors(cfg)
    assert {k: tuple(v.shape) for k, v in t.items()} == O.tensor_shapes(raw)
    w = map_torutar_weights(cfg, t, "cpu", torch.float32)
    a = w.layers[0].mix                                              # [q 48 | k 16 | v 10 | pad | g 6 | pad]
    assert aligned_columns(74, 6) == [0, 80, 88] and a["in"].shape == (88, 20)
    assert torch.equal(a["in"][64:74], t["l0.mix.v"].float()) and torch.equal(a["in"][80:86], t["l0.mix.g"].float())
    assert a["in"][74:80].abs().max() == 0 and a["in_b"][74:].abs().max() == 0
    assert torch.equal(a["in_b"][48:64], t["l0.mix.k.b"].float())
    shared = w.layers[3].mix
    assert shared["in"].shape == (56, 20) and "k_norm" not in shared
    q0, k0, v0, g0, i0, f0, end = aligned_columns(12, 12, 21, 21, 3, 3)
    m = w.layers[1].mix["in"]
    assert m.shape == (end, 20) and torch.equal(m[f0:f0 + 3], t["l1.mix.f"].float()) and torch.equal(m[g0:g0 + 21], t["l1.mix.g"].float())
    e = w.layers[0].mlp["gate_up"]                                   # gate and up rows of an expert interleave
    assert e.shape == (5, 12, 20) and torch.equal(e[3, 0::2], t["l0.mlp.e3.gate"].float()) and torch.equal(e[3, 1::2], t["l0.mlp.e3.up"].float())
    s = w.layers[0].subs
    assert len(s) == 2 and len(w.layers[1].subs) == 1
    assert torch.equal(s[1]["coef"][3:].view(3, 3), t["l0.hc2.mix"].float()) and s[0]["in"].dtype == torch.float32
    assert w.nbytes_per_step() > 0
    del t["l2.mix.uk"]
    with pytest.raises(KeyError):
        map_torutar_weights(cfg, t, "cpu", torch.float32)


def test_state_slots_hold_a_tail_per_sublayer():
    cfg = parse_torutar_config(_config())
    st = RecurrentStateManager(cfg, 4, torch.bfloat16, "cpu")
    assert set(st.input_tail) == {(0, 0), (0, 1), (1, 0), (2, 0), (2, 1), (3, 0)}
    assert all(x.shape == (4, 4, 20) and x.dtype == torch.bfloat16 for x in st.input_tail.values())
    assert st.ssm_state[1].shape == (4, 3, 36) and st.ssm_state[1].dtype == torch.float32
    assert st.nbytes() == 6 * 4 * 4 * 20 * 2 + 4 * 3 * 36 * 4


def test_rows_between_the_kept_tokens_and_the_windows_go_back():
    from lite_llama_b200.executor.model_runner import ModelRunner

    raw = O.make_config([O.attention_layer(size=10, keep_first=3), O.attention_layer(size=30, keep_first=7, kv_from=0)])
    cfg = parse_torutar_config(raw)
    w = map_torutar_weights(cfg, random_torutar_tensors(cfg), "cpu", torch.float32)
    runner = ModelRunner(cfg, w, 128, device="cpu", dtype=torch.float32, max_requests=2)
    assert runner.keep_positions == 29 + 64 and runner.keep_first == 7 and list(runner.kv_buffer_of) == [0]
    req = runner.open_request()
    for n in range(1, 400):                                          # what a step does to the pool, without its kernels
        req.rows.extend(runner.kv_cache_manager.alloc_rows_host(1))
        req.num_cached = n
        runner._release_unseen_rows(req)
        first, seen = req.rows[:min(n, 7)], req.rows[max(0, n - 30):]
        held = runner._held_rows(req)
        assert set(first) <= set(held) and set(seen) <= set(held) and len(set(held)) == len(held) == runner.rows_held(req)
        assert len(held) <= 93 + 7 and len(held) + runner.kv_cache_manager.can_use_mem_size == 128
    runner.close_request(req)
    assert runner.kv_cache_manager.can_use_mem_size == 128


# ------------------------------------------------------------------------------- the restatement's own invariants #
def test_a_layer_of_its_own_keys_equals_one_that_borrows_them():
    a = O.attention_layer(mlp=None)
    own, borrow = O.make_config([a, a], streams=2), O.make_config([a, dict(a, mixer=dict(a["mixer"], kv_from=0))], streams=2)
    w = O.random_model(own, 3)
    # layer 0 leaves the streams as they are and both layers read them alike, so both see the same keys
    for q in ("in", "mix"):
        w[f"l1.hc1.{q}"] = w[f"l0.hc1.{q}"]
    w["l0.hc1.out"] = torch.zeros(2)
    w["l0.hc1.mix"] = torch.eye(2)
    for name in list(w):
        if name.startswith("l0.mix.") and name.split("mix.")[1].split(".")[0] in ("k", "v") or name in ("l0.norm1", "l0.canon1"):
            w[name.replace("l0.", "l1.", 1)] = w[name]
    toks = [3, 9, 1, 1, 40, 7, 22, 5, 30, 2, 8]
    np.testing.assert_allclose(O.forward(own, w, toks), O.forward(borrow, w, toks), atol=1e-10)


def test_kept_tokens_windows_and_the_log_scale():
    assert [j for j in range(8) if O.sees(6, j, {"size": 2, "keep_first": 3})] == [0, 1, 2, 5, 6]
    assert [j for j in range(8) if O.sees(1, j, {"size": 1, "keep_first": 3})] == [0, 1]
    # the running scale only re-scales: a memory without it (m = 0 throughout) gives the same read-outs away from the floor
    m, rng = {"heads": 1, "dim": 3, "vdim": 2, "gate_cap": 4.0}, np.random.default_rng(0)
    w = {n: rng.standard_normal((r, 5)) for n, r in (("q", 3), ("k", 3), ("v", 2), ("g", 2), ("i", 1), ("f", 1))}
    w.update({"i.b": np.array([3.0]), "f.b": np.array([1.0]), "norm": np.ones(2), "o": np.eye(2)})
    h = rng.standard_normal((9, 5))
    S, n, got = np.zeros((3, 2)), np.zeros(3), []
    for x in h:
        gi = 4 * np.tanh((w["i"] @ x + 3.0) / 4)[0]
        gf = O.log_logistic(4 * np.tanh((w["f"] @ x + 1.0) / 4))[0]
        k, v, q = w["k"] @ x, w["v"] @ x, w["q"] @ x * 3 ** -0.5
        S, n = np.exp(gf) * S + np.exp(gi) * np.outer(k, v), np.exp(gf) * n + np.exp(gi) * k
        y = S.T @ q / max(abs(n @ q), 1.0)
        got.append(O.unit_rms(y, 1e-12) * O.logistic(w["g"] @ x))
    np.testing.assert_allclose(O.mlstm(h, m, w, 1e-12), np.stack(got), atol=1e-4)
