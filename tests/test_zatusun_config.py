"""Zatusun without a GPU: the configuration, the model description and its tensor names, what each layer asks of the
cache, and the plain restatement checked against second formulations of its mechanisms."""

import copy
import math

import numpy as np
import pytest

import plain_zatusun as S
import tiny_zatusun as tiny


def _parse(cfg):
    from kv_cache_optimization_for_llm_b200.registry import resolve_architecture
    arch = resolve_architecture(cfg)
    return arch, arch.parse_config(cfg)


def test_description_names_every_tensor_and_repeats_layers():
    arch, cfg = _parse(tiny.MIXED)
    spec = arch.build_spec(cfg)
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 3, 1, 2, 3, 4, 5] and all(e.cache_of is None for e in spec.schedule)
    assert [i for i, e in enumerate(spec.schedule) if e.before is not None] == [1, 4]
    assert [spec.schedule[i].before.params["index"] for i in (1, 4)] == [0, 1]
    assert [layer.block for layer in spec.layers] == ["prenorm", "prenorm", "prenorm_mixer_only", "prenorm",
                                                      "prenorm_mixer_only", "prenorm"]
    names = tiny.expected(tiny.MIXED)
    assert names["embed"].shape == (97, 40) and names["pos"].shape == (192, 40) and names["head"].shape == (97, 40)
    assert names["loop.in"].shape == (40, 80) and names["loop.step"].shape == (2, 40) and names["final.norm"].shape == (40,)
    assert names["l0.mix.q"].shape == (36, 40) and names["l0.mix.f"].shape == (36, 40) and names["l0.mix.f.b"].shape == (36,)
    assert names["l0.mix.lower"].shape == (36,) and names["l0.mix.v"].shape == (60, 40) and names["l0.mix.norm"].shape == (20,)
    assert names["l1.mix.q"].shape == (128, 40) and names["l1.mix.k"].shape == (64, 40) and names["l1.mix.v"].shape == (48, 40)
    assert names["l1.mix.lq2"].shape == (16,) and names["l1.mix.o"].shape == (40, 96)
    assert names["l2.mix.uq"].shape == (72, 20) and names["l2.mix.dkv"].shape == (32, 40) and names["l2.mix.uk"].shape == (48, 24)
    assert names["l2.mix.uv"].shape == (72, 24) and names["l2.mix.g"].shape == (72, 40) and names["l2.mix.dq.norm"].shape == (20,)
    assert "l2.mix.sink" not in names and "l2.norm2" not in names and "l4.norm1" in names
    assert names["l0.mlp.router"].shape == (5, 40) and names["l0.mlp.e4.gate"].shape == (12, 40)
    assert names["l1.mlp.e2.down"].shape == (40, 16) and not any(n.startswith(("l4.mlp", "l6.")) for n in names)


def test_what_the_parts_are_given():
    arch, cfg = _parse(tiny.MIXED)
    spec = arch.build_spec(cfg)
    att, lat = spec.layers[1].parts["mixer"].params, spec.layers[2].parts["mixer"].params
    assert att["chunk"] == 11 and att["diff"] == 0.4 and att["position"].params["scaling"]["rope_type"] == "llama3"
    assert lat["gate"] and not lat["sink"] and lat["position"].params["scaling"]["rope_type"] == "yarn"
    ff = spec.layers[0].parts["feed_forward"].params
    assert ff["score"] == "softmax_chosen" and ff["weigh"] == "output" and ff["shared_ff"] == 0 and ff["alpha"] == 1.702
    assert spec.embedding.params["scale"] == 3.0 and spec.lm_head.params["softcap"] == 7.0 and spec.max_position == 192


def test_what_the_config_leaves_out_is_not_there():
    cfg = tiny.config([tiny.layer("attention", tiny.attention(size=None, rot_dims=None)),
                       tiny.layer("latent_attention", tiny.latent(scaling=None))], logit_softcap=None)
    arch, parsed = _parse(cfg)
    spec = arch.build_spec(parsed)
    att = spec.layers[0].parts["mixer"].params
    assert att["chunk"] is None and att["position"] is None and spec.lm_head.params["softcap"] is None
    assert spec.layers[1].parts["mixer"].params["position"].params["scaling"] is None
    assert all(e.before is None for e in spec.schedule) and "loop.in" not in tiny.expected(cfg)


def test_positions_may_be_left_to_the_tables_shape():
    from kv_cache_optimization_for_llm_b200.config import ConfigError
    cfg = copy.deepcopy(tiny.MIXED)
    del cfg["max_positions"]
    arch, parsed = _parse(cfg)
    assert arch.build_spec(arch.complete(parsed, {"pos": (77, 40)})).max_position == 77
    with pytest.raises(ConfigError, match="max_positions"):
        arch.build_spec(parsed)


@pytest.mark.parametrize("breakage,needle", [
    (lambda c: c["layers"][1]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][2]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "grouped"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=10), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(scaling={"factor": 2.0, "original": 9, "slow": 1.0}), "fast"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(scaling={"factor": 2.0, "original": 9, "low": 1.0}), "high"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "dense"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "top"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][0].update(type="conv"), "conv"),
    (lambda c: c["loop"].update(stop=9), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["loop"].update(start=4), "loop"),
    (lambda c: c.pop("width"), "width"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_config_errors_name_the_key(breakage, needle):
    from kv_cache_optimization_for_llm_b200.config import ConfigError
    cfg = copy.deepcopy(tiny.MIXED)
    breakage(cfg)
    with pytest.raises(ConfigError) as e:
        _parse(cfg)
    assert needle in str(e.value)


def test_the_engines_frequencies_are_the_plain_ones():
    from kv_cache_optimization_for_llm_b200.parts.position import rope_inv_freq, yarn_inv_freq
    for dims, base, sc in ((10, 500.0, tiny.YARN), (64, 1e4, dict(factor=8.0, original=512, fast=32.0, slow=1.0)),
                           (2, 3.0, dict(factor=1.5, original=7, fast=2.0, slow=1.0))):
        f, grow = S.ramped_frequencies(dims, base, sc["factor"], sc["original"], sc["fast"], sc["slow"])
        g, grow2 = yarn_inv_freq(dims, base, sc)
        assert np.abs(g.numpy() - f).max() < 1e-15 and abs(grow - grow2) < 1e-15
    for dims, base, sc in ((24, 300.0, tiny.BANDS), (64, 5e5, dict(factor=8.0, original=300, low=1.0, high=4.0)), (2, 9.0, tiny.BANDS)):
        f = S.banded_frequencies(dims, base, sc["factor"], sc["low"], sc["high"], sc["original"])
        g = rope_inv_freq(dims, base, {"rope_type": "llama3", "factor": sc["factor"], "low_freq_factor": sc["low"],
                                       "high_freq_factor": sc["high"], "original_max_position_embeddings": sc["original"]})
        assert np.abs(g.numpy() - f).max() < 1e-15


def test_banded_frequencies_keep_short_waves_divide_long_ones_and_blend_between():
    dims, base, sc = 32, 1e4, dict(factor=4.0, low=1.0, high=4.0, original=200)
    plain = S.plain_frequencies(dims, base)
    ratio = plain / S.banded_frequencies(dims, base, **sc)
    wave = 2 * math.pi / plain
    assert np.all(ratio[wave < 50] == 1.0) and np.all(np.abs(ratio[wave > 200] - 4.0) < 1e-12)
    mid = (wave > 50) & (wave < 200)
    assert mid.sum() >= 2 and np.all((ratio[mid] > 1.0) & (ratio[mid] < 4.0)) and np.all(np.diff(ratio) >= -1e-12)


def test_rotation_depends_on_the_distance_only_and_pairs_neighbours():
    rng = np.random.default_rng(0)
    f = S.plain_frequencies(6, 50.0)
    q, k = rng.normal(size=(1, 1, 8)), rng.normal(size=(1, 1, 8))
    a = S.rotate_pairs(q, [17], f)[0, 0] @ S.rotate_pairs(k, [12], f)[0, 0]
    assert abs(a - S.rotate_pairs(q, [105], f)[0, 0] @ S.rotate_pairs(k, [100], f)[0, 0]) < 1e-12
    z = q[0, 0, 2] + 1j * q[0, 0, 3]
    turned = S.rotate_pairs(q, [9], f, 1.5)[0, 0]
    assert abs(turned[2] + 1j * turned[3] - z * 1.5 * np.exp(9j * f[1])) < 1e-12 and np.array_equal(turned[6:], q[0, 0, 6:])


def test_blocks_of_positions_are_counted_from_the_start():
    seen = [[j for j in range(12) if S.same_block(i, j, 5)] for i in range(12)]
    assert seen[4] == [0, 1, 2, 3, 4] and seen[5] == [5] and seen[9] == [5, 6, 7, 8, 9] and seen[11] == [10, 11]
    assert [j for j in range(4) if S.same_block(3, j, None)] == [0, 1, 2, 3]


def test_two_maps_are_subtracted_before_the_norm():
    """One query over two keys whose weights are known: a1 picks the first value, a2 mixes both evenly."""
    k = np.array([[[[1.0], [1.0]]], [[[-1.0], [1.0]]]])                   # [T, G, map, D]
    q = np.zeros((2, 1, 2, 1))
    q[1, 0, 0, 0] = 40.0
    v = np.array([[[3.0, 0.0]], [[0.0, 1.0]]])
    out = S.two_map_attention(q, k, v, 1.0, None, 0.5, 0.2, 0.0)[1, 0]
    d = np.array([3.0, 0.0]) - 0.5 * np.array([1.5, 0.5])
    assert np.abs(out - 0.8 * d / math.sqrt((d * d).mean())).max() < 1e-12
    w = {"lq1": np.array([1.0, 2.0]), "lk1": np.array([0.5, -0.25]), "lq2": np.array([0.3, 0.0]), "lk2": np.array([2.0, 7.0])}
    assert abs(S.difference_weight(w, "", 0.25) - (1.0 - math.exp(0.6) + 0.25)) < 1e-12


def test_memory_is_a_sum_over_the_past_with_products_of_decays():
    rng = np.random.default_rng(1)
    T, N, Dv = 7, 4, 3
    q, v, f = rng.normal(size=(T, N)), rng.normal(size=(T, Dv)), rng.uniform(0.1, 0.99, size=(T, N))
    got = S.decayed_memory(q, f, v)
    for t in range(T):
        ref = sum(((q[t] * np.prod(f[s + 1:t + 1], axis=0)) @ (1.0 - f[s])) * v[s] for s in range(t + 1))
        assert np.abs(got[t] - ref).max() < 1e-12
    assert np.allclose(S.decayed_memory(q, np.ones_like(f), v), 0.0)          # a gate of one writes nothing
    assert np.allclose(S.decayed_memory(q, np.zeros_like(f), v), q.sum(1, keepdims=True) * v)      # a gate of zero keeps nothing


def test_latent_attention_is_attention_over_absorbed_queries():
    rng = np.random.default_rng(2)
    m, W, T = tiny.latent(heads=2, dim=4, rot_dim=2, vdim=3, q_rank=5, kv_rank=6), 7, 9
    shapes = {"dq": (5, W), "dq.norm": (5,), "uq": (12, 5), "dkv": (8, W), "dkv.norm": (6,), "uk": (8, 6), "uv": (6, 6), "g": (6, W),
              "o": (W, 6)}
    w = {k: rng.normal(size=s) for k, s in shapes.items()}
    h = rng.normal(size=(T, W))
    got = S.latent_attention_mixer(h, w, "", m, 1e-5)
    c = S.rms_norm((h @ w["dkv"].T)[:, :6], w["dkv.norm"], 1e-5)
    f, grow = S.ramped_frequencies(2, m["rot"]["base"], **m["rot"]["scaling"])
    kr = S.rotate_pairs((h @ w["dkv"].T)[:, 6:], range(T), f, grow)
    q = (S.rms_norm(h @ w["dq"].T, w["dq.norm"], 1e-5) @ w["uq"].T).reshape(T, 2, 6)
    qr = S.rotate_pairs(q[:, :, 4:], range(T), f, grow)
    heads = []
    for a in range(2):
        absorbed = q[:, a, :4] @ w["uk"][4 * a:4 * a + 4]
        p = S.softmax_rows((absorbed @ c.T + qr[:, a] @ kr.T) * m["scale"], np.tril(np.ones((T, T), bool)))
        heads.append(p @ c @ w["uv"][3 * a:3 * a + 3].T)
    ref = (np.concatenate(heads, axis=1) * S.sigmoid(h @ w["g"].T)) @ w["o"].T
    assert np.abs(got - ref).max() < 1e-12


def test_experts_are_weighed_on_their_output_by_a_softmax_over_the_chosen():
    rng = np.random.default_rng(3)
    W, F = 6, 5
    w = {"router": rng.normal(size=(4, W))}
    for e in range(4):
        w.update({f"e{e}.gate": rng.normal(size=(F, W)), f"e{e}.up": rng.normal(size=(F, W)), f"e{e}.down": rng.normal(size=(W, F))})
    h = rng.normal(size=(3, W))
    chosen, weight = S.route(h, w["router"], 2)
    assert np.abs(weight.sum(1) - 1.0).max() < 1e-12 and np.all(weight[:, 0] >= weight[:, 1])
    out = S.moe(h, w, "", tiny.moe(experts=4, top=2, ff=F, limit=0.7))
    z = np.exp(h[1] @ w["router"].T)
    a, b = chosen[1]
    y = [S.limited_expert(h[1][None], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], 0.7)[0] for e in (a, b)]
    assert np.abs(out[1] - (z[a] * y[0] + z[b] * y[1]) / (z[a] + z[b])).max() < 1e-12
    # one chosen expert: its weight is 1 whatever its logit
    assert np.all(S.route(h, w["router"], 1)[1] == 1.0)


def test_every_pass_starts_from_the_stream_and_the_embedding():
    cfg = tiny.config([tiny.layer("hgrn2", tiny.hgrn2(heads=1, dim=2, vdim=2)) for _ in range(3)], width=4, vocab=5, loop=(0, 2, 3))
    assert S.layer_runs(cfg) == [(0, 0), (1, None), (0, 1), (1, None), (0, 2), (1, None), (2, None)]
    rng = np.random.default_rng(4)
    w = {"loop.in": rng.normal(size=(4, 8)), "loop.step": rng.normal(size=(3, 4))}
    x, x0 = rng.normal(size=(2, 4)), rng.normal(size=(2, 4))
    assert np.abs(S.start_pass(x, x0, w, 1) - (x @ w["loop.in"][:, :4].T + x0 @ w["loop.in"][:, 4:].T + w["loop.step"][1])).max() < 1e-12
