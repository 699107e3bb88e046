"""Host side of the Povilorn design: configuration parser, registry, loop unrolling, weight mapping, cache shapes, and the
restatement's own invariants.  No GPU."""

from __future__ import annotations

import math

import numpy as np
import pytest
import torch

import povilorn_oracle as O
from lite_llama_b200.executor.layered_decoder import (aligned_columns, looped_order, map_povilorn_weights,
                                                      parse_povilorn_config, povilorn_tensor_shapes, random_povilorn_tensors)
from lite_llama_b200.executor.model_config import DenseMlpSpec, LatentAttentionSpec, MoeMlpSpec, SinkAttentionSpec
from lite_llama_b200.executor.registry import lookup
from lite_llama_b200.kernels import key_factor_column, rotary_frequencies


def _config():
    return O.make_config([O.latent_layer(heads=3, dim=5, rot_dim=6, vdim=4, kv_rank=7, base=777.0, scale=0.3,
                                         scaling={"factor": 3.0, "original": 50, "fast": 8.0, "slow": 0.25}),
                          O.attention_layer(heads=6, kv_heads=2, dim=5, coef=0.7, every=11, scale=0.4,
                                            mlp=O.moe_mlp(7, 5, 3, 6, 0.8, 3, 2, 5, 0.5)),
                          O.attention_layer(heads=4, kv_heads=4, dim=8, every=0, mlp=None),
                          O.latent_layer(scaling=False, mlp=O.moe_mlp(4, 0, 2, 3, shared_ff=0))],
                         width=20, vocab=33, eps=1e-4, embed_scale=2.5, loop=(1, 3, 2))


def test_every_size_and_constant_comes_from_the_configuration():
    cfg = lookup("povilorn").parse_config(_config())
    cfg.validate()
    assert (cfg.hidden_size, cfg.vocab_size, cfg.embed_scale, cfg.rms_norm_eps, cfg.max_seq_len, cfg.norm_kind, cfg.loop_passes) == \
        (20, 33, 2.5, 1e-4, 0, "tanh", 2)
    assert [l.source for l in cfg.layers] == [0, 1, 2, 1, 2, 3]
    assert [l.weights_of for l in cfg.layers] == [None, None, None, 1, 2, None]
    assert [l.loop_pass for l in cfg.layers] == [None, 0, None, 1, None, None]
    l, a, b = (cfg.layers[i].mixer for i in (0, 1, 2))
    assert isinstance(l, LatentAttentionSpec) and (l.heads, l.head_dim, l.rot_dim, l.v_head_dim, l.q_rank, l.kv_rank) == (3, 5, 6, 4, 0, 7)
    assert (l.scale, l.rot_dims, l.rot_base, l.rot_factor, l.rot_original, l.rot_fast, l.rot_slow) == (0.3, 6, 777.0, 3.0, 50, 8.0, 0.25)
    assert l.pairing == "neighbours" and not l.out_gate and l.window == 0
    assert isinstance(a, SinkAttentionSpec) and (a.heads, a.kv_heads, a.head_dim, a.v_head_dim) == (6, 2, 5, 5)
    assert (a.scale, a.gain_coef, a.gain_every, a.keys_as_values, a.element_gate) == (0.4, 0.7, 11.0, True, True)
    assert b.gain_every == 0.0 and cfg.layers[5].mixer.rot_factor == 1.0
    d, m, n = cfg.layers[0].mlp, cfg.layers[1].mlp, cfg.layers[5].mlp
    assert isinstance(d, DenseMlpSpec) and (d.ff, d.activation, d.gated) == (9, "gelu_tanh", True)
    assert isinstance(m, MoeMlpSpec) and (m.experts, m.identity, m.choices, m.top, m.ff, m.limit) == (7, 5, 12, 3, 6, 0.8)
    assert (m.groups, m.keep, m.group_score, m.scores, m.activation, m.renormalize, m.alpha) == (3, 2, "max", "softmax", "clamped", True, 1.702)
    assert (m.shared_ff, m.shared_limit, m.shared_gate) == (5, 0.5, True)
    assert (n.identity, n.shared_ff, n.shared_gate) == (0, 0, False) and cfg.layers[2].mlp is None
    assert cfg.attention_layers() == [0, 1, 2, 3, 4, 5]                # every run of a looped layer has a cache of its own


@pytest.mark.parametrize("count,loop,order", [
    (3, None, [(0, None), (1, None), (2, None)]),
    (3, {"start": 0, "stop": 3, "times": 1}, [(0, 0), (1, None), (2, None)]),
    (4, {"start": 1, "stop": 2, "times": 3}, [(0, None), (1, 0), (1, 1), (1, 2), (2, None), (3, None)]),
    (4, {"start": 2, "stop": 4, "times": 2}, [(0, None), (1, None), (2, 0), (3, None), (2, 1), (3, None)])])
def test_loops_unroll_in_place(count, loop, order):
    assert looped_order(count, loop) == order
    assert O.run_order({"layers": [{}] * count, "loop": loop}) == order


@pytest.mark.parametrize("break_it", [lambda c: c["layers"][0].update(type="lstm"), lambda c: c["layers"][0]["mlp"].update(kind="maxout"),
                                      lambda c: c["layers"][1]["mixer"].update(kv_heads=4), lambda c: c["layers"][1]["mixer"].update(vdim=4),
                                      lambda c: c["layers"][1]["mlp"]["router"].update(top=9),
                                      lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=5),
                                      lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4),
                                      lambda c: c["layers"][0]["mixer"]["rot"].update(dims=5),
                                      lambda c: c["loop"].update(stop=5), lambda c: c["loop"].update(start=3), lambda c: c["loop"].update(times=0)])
def test_what_does_not_fit_is_refused(break_it):
    raw = _config()
    break_it(raw)
    with pytest.raises(ValueError):
        parse_povilorn_config(raw).validate()


def test_names_shapes_and_layouts_of_the_weights():
    raw = _config()
    cfg = parse_povilorn_config(raw)
    assert povilorn_tensor_shapes(cfg) == O.tensor_shapes(raw)
    t = random_povilorn_tensors(cfg)
    assert {k: tuple(v.shape) for k, v in t.items()} == O.tensor_shapes(raw)
    w = map_povilorn_weights(cfg, t, "cpu", torch.float32)
    a = w.layers[1].mix                                              # [q 30 | k 10 | g 30 | pad]
    assert aligned_columns(40, 30) == [0, 40, 72] and a["qkv"].shape == (72, 20)
    assert torch.equal(a["qkv"][30:40], t["l1.mix.k"].float()) and torch.equal(a["qkv"][40:70], t["l1.mix.g"].float())
    assert torch.equal(a["qkv_b"][30:40], t["l1.mix.k.b"].float()) and a["qkv_b"][40:].abs().max() == 0
    qw, kw = t["l1.mix.q.norm"].float().view(6, 5), t["l1.mix.k.norm"].float().view(2, 5)
    assert a["query_weight"].dtype == torch.float32
    for h in range(6):
        assert torch.equal(a["query_weight"].view(6, 5)[h], qw[h] * kw[h // 3])
    l = w.layers[0].mix                                              # [q 33 | pad | latent 7 | rotated 6 | pad]
    assert l["down"].shape == (56, 20) and torch.equal(l["down"][40:53], t["l0.mix.dkv"].float())
    assert l["down"][33:40].abs().max() == 0 and l["freqs"].dtype == torch.float64 and l["freqs"].numel() == 3
    assert w.layers[3] is w.layers[1] and w.layers[4] is w.layers[2] and w.loop_step.shape == (2, 20)
    e = w.layers[1].mlp["gate_up"]                                   # gate and up rows of an expert interleave
    assert e.shape == (7, 12, 20) and torch.equal(e[3, 0::2], t["l1.mlp.e3.gate"].float()) and torch.equal(e[3, 1::2], t["l1.mlp.e3.up"].float())
    s = w.layers[1].mlp["shared_gate_up"]
    assert s.shape == (16, 20) and torch.equal(s[10], t["l1.mlp.shared.sg"].float()[0]) and s[11:].abs().max() == 0
    assert w.layers[1].mlp["router"].shape == (12, 20)
    assert w.layers[1].subs[1]["alpha"].shape == (1,) and torch.equal(w.final_sub["norm_b"], t["final.norm.b"].float())
    assert len(w.layers[2].subs) == 1 and w.nbytes_per_step() > 0
    del t["l3.mix.uk"]
    with pytest.raises(KeyError):
        map_povilorn_weights(cfg, t, "cpu", torch.float32)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_cache_rows_hold_the_keys_once_and_their_statistic(dtype):
    from lite_llama_b200.executor.model_runner import ModelRunner

    cfg = parse_povilorn_config(_config())
    w = map_povilorn_weights(cfg, random_povilorn_tensors(cfg), "cpu", dtype)
    runner = ModelRunner(cfg, w, 128, device="cpu", dtype=dtype, max_requests=2)
    widths = {i: b.shape[1] for i, b in runner.kv_buffer_of.items()}
    assert widths == {0: 16, 1: 16, 2: 40, 3: 16, 4: 40, 5: 16}      # 7 + 6, 2 * 5 + statistic, 4 * 8 + statistic, ..., 6 + 4
    assert len({b.data_ptr() for b in runner.kv_buffer_of.values()}) == 6
    for keys in range(1, 70):
        width = SinkAttentionSpec(1, 1, keys, keys, 1.0, keys_as_values=True).cache_row_width
        assert width % 8 == 0 and keys <= key_factor_column(keys) <= width - 2 and key_factor_column(keys) % 2 == 0


# ------------------------------------------------------------------------------- the restatement's own invariants #
def test_a_folded_key_norm_scores_like_the_normed_key():
    """q . (k / rms(k) * wk) = ((q * wk) . k) / rms(k): the identity the cache row rests on."""
    rng = np.random.default_rng(0)
    q, k, wk = rng.standard_normal((3, 12))
    normed = O.unit_rms(k, 1e-5) * wk
    assert abs(q @ normed - (q * wk) @ k / math.sqrt(np.mean(k * k) + 1e-5)) < 1e-12


def test_interpolated_frequencies_agree_with_the_framework():
    for dims, base, sc in ((6, 777.0, {"factor": 3.0, "original": 50, "fast": 8.0, "slow": 0.25}),
                           (64, 1e4, {"factor": 16.0, "original": 4096, "fast": 32.0, "slow": 1.0}),
                           (8, 100.0, {"factor": 2.0, "original": 10, "fast": 1.0, "slow": 1.0})):
        ours, mag = O.rotation_plan(dims, base, sc)
        theirs, mag2 = rotary_frequencies(dims, base, sc["factor"], sc["original"], sc["fast"], sc["slow"])
        np.testing.assert_allclose(ours, theirs, rtol=1e-13)
        assert mag == mag2 and mag > 1.0
        assert ours[0] >= ours[-1] and any(abs(a - base ** (-2 * i / dims)) > 1e-9 for i, a in enumerate(ours))


def test_groups_corrections_and_identity_experts_in_the_choice():
    w = {"router": np.eye(6), "correction": np.array([-0.9, -0.9, -0.9, -0.9, 0.0, 0.0])}
    r = {"experts": 4, "identity": 2, "top": 2, "groups": {"count": 3, "keep": 1}}
    pick, weights = O.choose(np.array([3.0, 2.0, 1.0, 0.0, -1.0, -2.0]), r, w)
    assert sorted(pick) == [4, 5] and abs(weights.sum() - 1) < 1e-12       # negative choice scores lose to the identities
    r["groups"] = {"count": 3, "keep": 2}
    r["top"] = 3
    pick, _ = O.choose(np.array([3.0, 2.0, 1.0, 0.0, -1.0, -2.0]), r, w)
    assert list(pick) == [4, 5, 0]                                         # and a kept group's negative score still beats -inf
    # a group wins by its best member, not by its sum
    pick, _ = O.choose(np.array([3.0, -9.0, 2.8, 2.8, 0.0, 0.0]), dict(r, top=1, groups={"count": 3, "keep": 1}),
                       {"router": np.eye(6)})
    assert list(pick) == [0]


def test_the_first_pass_of_a_loop_adds_its_vector_and_later_ones_the_embedding_too():
    layer = O.attention_layer(mlp=None)
    cfg = O.make_config([layer], loop=(0, 1, 3))
    w = O.random_model(cfg, 3)
    w["l0.mix.o"] = w["l0.mix.o"] * 0                                      # the layer adds nothing: what is left is the loop
    x = O.f64(w["embed"])[[4, 9]] * 3.0
    _, layers = O.forward(cfg, w, [4, 9], return_layers=True)
    steps = O.f64(w["loop.step"])
    for t in range(3):
        np.testing.assert_allclose(layers[t], (t + 1) * x + steps[:t + 1].sum(0), atol=1e-12)
