"""Lobuzen without a GPU: the configuration, the model description and its tensor names, what each layer asks of the
cache, and the plain restatement checked against second formulations of its mechanisms."""

import copy

import numpy as np
import pytest
import torch

import plain_lobuzen as S
import tiny_lobuzen as tiny


def _parse(cfg):
    from kv_cache_optimization_for_llm_b200.registry import resolve_architecture
    arch = resolve_architecture(cfg)
    return arch, arch.parse_config(cfg)


def _spec(cfg):
    arch, parsed = _parse(cfg)
    return arch.build_spec(parsed)


def test_description_names_every_tensor():
    spec = _spec(tiny.MIXED)
    assert [e.layer for e in spec.schedule] == list(range(6))
    assert [e.cache_of for e in spec.schedule] == [None, None, 0, 0, None, None]
    assert [x.block for x in spec.layers] == ["postnorm_token_input"] * 3 + ["postnorm_token_input_mixer_only"] + ["postnorm_token_input"] * 2
    names = tiny.expected(tiny.MIXED)
    assert names["embed"].shape == (97, 48) and names["side.embed"].shape == (97, 48) and "head" not in names
    assert names["l0.mix.q"].shape == (48, 48) and names["l0.mix.dkv"].shape == (40, 48) and names["l0.mix.dkv.norm"].shape == (40,)
    assert names["l0.mix.uk"].shape == (48, 40) and names["l0.mix.uv"].shape == (72, 40) and names["l0.mix.sink"].shape == (3,)
    assert names["l2.mix.uk"].shape == (40, 40) and names["l2.mix.uv"].shape == (80, 40) and names["l2.mix.o"].shape == (48, 80)
    assert not any(n.startswith(("l2.mix.dkv", "l3.mix.dkv", "l3.mlp", "l6.")) for n in names) and "l3.norm2" not in names
    assert names["l1.mix.k"].shape == (48, 48) and names["l1.mix.v"].shape == (72, 48) and "l1.mix.q_norm" not in names
    assert names["l0.mlp.up"].shape == (56, 48) and names["l2.mlp.e7.down"].shape == (48, 12) and names["l2.mlp.correction"].shape == (8,)
    assert names["l3.side.gate"].shape == (8, 48) and names["l3.side.proj"].shape == (48, 8) and names["l3.side.norm"].shape == (48,)


def test_what_the_parts_are_given():
    spec = _spec(tiny.MIXED)
    own, borrowed, att = (spec.layers[i].parts["mixer"].params for i in (0, 2, 1))
    assert own["window"] == 19 and own["sink"] and not own["borrows_latent"] and not own["q_rank"] and own["rot_dim"] == 0
    assert borrowed["window"] == 33 and borrowed["borrows_latent"]
    assert att["qk_norm"] == "unweighted" and att["window"] == 11
    ff, grouped, free = (spec.layers[i].parts["feed_forward"].params for i in (0, 2, 5))
    assert ff["limit"] == 1.1 and ff["alpha"] == 1.702 and ff["offset"] == 1.0
    assert (grouped["groups"], grouped["keep_groups"]) == (4, 2) and free["groups"] == 0
    assert grouped["limit"] is None and grouped["offset"] == 0.0 and grouped["alpha"] == 1.0 and grouped["weigh"] == "output"
    assert [x.parts["token_input"].params["first"] for x in spec.layers] == [0, 8, 16, 24, 32, 40]


def test_what_the_config_leaves_out_is_not_there():
    cfg = tiny.config([tiny.layer("attention", tiny.attention(size=None)),
                       tiny.layer("latent_attention", tiny.latent(size=None), tiny.moe(groups=None))], side=None)
    spec = _spec(cfg)
    assert [x.block for x in spec.layers] == ["postnorm_mixer_only", "postnorm"]
    assert all(x.parts["mixer"].params["window"] is None for x in spec.layers)
    assert not any("side" in n for n in tiny.expected(cfg))


@pytest.mark.parametrize("breakage,needle", [
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "grouped"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=5), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_rank=32), "kv_rank"),
    (lambda c: c["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "sparse"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4), "groups"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].pop("keep"), "keep"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=3, groups={"count": 3, "keep": 1}), "top"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda c: c["layers"][0].update(type="conv"), "conv"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
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


# --------------------------------------------------------------------------- a cache that several layers read

def _cache(wishes, cache_of, pages=20):
    from kv_cache_optimization_for_llm_b200.cache.paged_cache import PagedCache
    return PagedCache(wishes, cache_of, 8, pages, 2, 256, torch.float32, "cpu")


def test_borrowed_rows_are_kept_as_long_as_the_reader_that_sees_furthest():
    from kv_cache_optimization_for_llm_b200.cache import PagedKVSpec
    row = lambda w: PagedKVSpec(1, 40, w, planes=1)
    c = _cache([row(19), row(33), row(6), row(19)], [None, 0, 0, None])
    # the owner's group is as wide as its widest reader; the same wish without readers is a group of its own
    assert [k[2] for k in c.group_keys] == [33, 19] and c.group_entries == [1, 1]
    owner, far, near = (c.binding(i) for i in (0, 1, 2))
    assert owner.write and not far.write and not near.write and far.k.data_ptr() == near.k.data_ptr() == owner.k.data_ptr()
    assert {b.group for b in (owner, far, near)} == {0}
    m = c.manager
    m.admit(1)
    m.extend(1, 60)
    m.advance(1, 60)
    # the next token sits at 60: keys from 28 on for a window of 33 (pages of 8: 24 .. ), from 42 on for one of 19
    assert [p < 0 for p in m.block_table(1, 0)] == [True] * 3 + [False] * 5
    assert [p < 0 for p in m.block_table(1, 1)] == [True] * 5 + [False] * 3
    m.release(1)
    assert m.check() == "" and m.free_pages(0) == m.free_pages(1) == 20


def test_a_reader_without_a_window_keeps_every_page_and_other_rows_are_refused():
    from kv_cache_optimization_for_llm_b200.cache import PagedKVSpec
    c = _cache([PagedKVSpec(1, 16, 5, planes=1), PagedKVSpec(1, 16, None, planes=1)], [None, 0])
    assert [k[2] for k in c.group_keys] == [0]
    with pytest.raises(ValueError, match="cannot read the cache"):
        _cache([PagedKVSpec(1, 16, 5, planes=1), PagedKVSpec(1, 24, 5, planes=1)], [None, 0])


# --------------------------------------------------------------------------- the plain model, a second time

def test_a_window_holds_the_last_positions_and_the_token_itself():
    seen = [[j for j in range(9) if S.in_window(i, j, 4)] for i in range(9)]
    assert seen[0] == [0] and seen[3] == [0, 1, 2, 3] and seen[4] == [1, 2, 3, 4] and seen[8] == [5, 6, 7, 8]
    assert [j for j in range(5) if S.in_window(3, j, 1)] == [3] and [j for j in range(5) if S.in_window(3, j, None)] == [0, 1, 2, 3]


def test_a_sink_is_a_key_with_that_score_and_a_value_of_zero():
    rng = np.random.default_rng(0)
    s, v, sink = rng.normal(size=(1, 5)) * 3, rng.normal(size=(5, 2)), 1.7
    seen = np.array([[False, True, True, True, False]])
    e = np.exp(np.append(s[0, 1:4], sink))
    ref = e[:3] @ v[1:4] / e.sum()
    assert np.abs(S.softmax_rows(s, seen, sink) @ v - ref).max() < 1e-14
    assert np.abs(S.softmax_rows(s, seen, -1e9) - S.softmax_rows(s, seen)).max() < 1e-14


def test_query_and_key_heads_are_divided_by_their_root_mean_square():
    rng = np.random.default_rng(1)
    m, W, T = tiny.attention(heads=2, kv_heads=1, dim=4, vdim=3, size=None), 6, 5
    w = {"q": rng.normal(size=(8, W)), "k": rng.normal(size=(4, W)), "v": rng.normal(size=(3, W)), "o": rng.normal(size=(W, 6))}
    h = rng.normal(size=(T, W))
    got = S.attention_mixer(h, w, "", m, 0.0)
    # without eps only the directions of queries and keys matter
    scaled = dict(w, q=np.concatenate([w["q"][:4] * 5.0, w["q"][4:] * 0.1]), k=w["k"] * 30.0)
    assert np.abs(S.attention_mixer(h, scaled, "", m, 0.0) - got).max() < 1e-12
    cos = [float(a @ b) / (np.linalg.norm(a) * np.linalg.norm(b)) for a, b in [(w["q"][:4] @ h[1], w["k"] @ h[j]) for j in (0, 1)]]
    e = np.exp(np.array(cos) * 4 * m["scale"])       # two unit-rms vectors of four channels: dot = 4 cos
    head0 = (e / e.sum()) @ (h[:2] @ w["v"].T)
    q, k, v = (S.rms_norm((h @ w["q"].T).reshape(T, 2, 4), None, 0.0), S.rms_norm((h @ w["k"].T).reshape(T, 1, 4), None, 0.0),
               (h @ w["v"].T).reshape(T, 1, 3))
    assert np.abs(S.attend(q, k, v, m["scale"], None)[1, 0] - head0).max() < 1e-12


def test_latent_attention_is_attention_over_absorbed_queries():
    rng = np.random.default_rng(2)
    m, W, T, R = tiny.latent(heads=2, dim=4, vdim=3, kv_rank=6, size=4), 7, 9, 6
    w = {"q": rng.normal(size=(8, W)), "dkv": rng.normal(size=(R, W)), "dkv.norm": rng.normal(size=(R,)), "uk": rng.normal(size=(8, R)),
         "uv": rng.normal(size=(6, R)), "sink": rng.normal(size=(2,)), "o": rng.normal(size=(W, 6))}
    h = rng.normal(size=(T, W))
    c = S.latent(h, w, "", 1e-5)
    heads = []
    for a in range(2):
        absorbed = (h @ w["q"][4 * a:4 * a + 4].T) @ w["uk"][4 * a:4 * a + 4]
        p = S.softmax_rows(absorbed @ c.T * m["scale"], S.in_window(np.arange(T)[:, None], np.arange(T)[None, :], 4), w["sink"][a])
        heads.append(p @ c @ w["uv"][3 * a:3 * a + 3].T)
    assert np.abs(S.latent_attention_mixer(h, c, w, "", m) - np.concatenate(heads, axis=1) @ w["o"].T).max() < 1e-12


def test_experts_are_chosen_through_their_groups_and_weighed_by_their_bare_scores():
    z = np.array([[4.0, -9.0, 1.0, 1.2, 2.0, -3.0]])               # logits, groups of two neighbours
    eye = np.eye(6)
    s = S.sigmoid(z[0])
    # group sums: s0 + s1 = 0.98, s2 + s3 = 1.50, s4 + s5 = 0.93: the largest score alone does not save its group
    chosen, weights = S.route(z, eye, np.zeros(6), 2, {"count": 3, "keep": 1})
    assert list(chosen[0]) == [3, 2] and np.allclose(weights[0], [s[3], s[2]])
    chosen, _ = S.route(z, eye, np.zeros(6), 2, {"count": 3, "keep": 2})
    assert list(chosen[0]) == [0, 3]
    assert list(S.route(z, eye, np.zeros(6), 2)[0][0]) == [0, 4]
    # the correction moves the choice, among groups and inside them, and leaves the weights alone; choice scores below zero
    # still beat an expert of a group that is out
    low = np.array([-3.0, -3.0, -2.0, -1.5, -9.0, -9.0])
    chosen, weights = S.route(z, eye, low, 2, {"count": 3, "keep": 1})
    assert list(chosen[0]) == [3, 2] and np.allclose(weights[0], [s[3], s[2]])
    chosen, weights = S.route(z, eye, np.array([0, 0, 0, 0, 5.0, 0]), 1, {"count": 3, "keep": 1})
    assert list(chosen[0]) == [4] and np.allclose(weights[0], [s[4]])
    # groups of one expert each are judged by that expert
    assert list(S.route(z, eye, np.zeros(6), 2, {"count": 6, "keep": 3})[0][0]) == [0, 4]


def test_limited_dense_and_the_tokens_own_input_by_hand():
    w = {"gate": np.array([[3.0], [0.5]]), "up": np.array([[-4.0], [0.25]]), "down": np.array([[1.0, 10.0]])}
    y = S.limited_dense(np.array([[1.0]]), w, "", {"limit": 2.0})
    a = 2.0 * S.sigmoid(1.702 * 2.0) * (-2.0 + 1.0), 0.5 * S.sigmoid(1.702 * 0.5) * 1.25
    assert abs(y[0, 0] - (a[0] + 10.0 * a[1])) < 1e-14
    w = {"gate": np.array([[1.0, 0.0]]), "proj": np.array([[3.0], [4.0]]), "norm": np.array([1.0, 2.0])}
    y = S.token_input(np.array([[1.5, 9.0]]), np.array([[-0.2]]), w, "", 0.0)
    assert np.abs(y[0] - np.array([-3.0, -8.0]) / np.sqrt(12.5)).max() < 1e-14      # only the sign of the gated row is left


def test_the_stream_is_read_bare_and_layers_take_their_own_columns_of_a_tokens_row():
    cfg = tiny.config([tiny.layer("attention", tiny.attention(heads=1, kv_heads=1, dim=2, vdim=2)) for _ in range(2)], width=4, vocab=5, side=3)
    w = {k: v.double().numpy() for k, v in tiny.draw_weights(cfg, 0).items()}
    toks = [1, 4, 2]
    z, after = S.forward(cfg, w, toks, keep_layers=True)
    x = w["embed"][toks]
    for i in range(2):
        p = f"l{i}."
        x = x + S.rms_norm(S.attention_mixer(x, w, p + "mix.", cfg["layers"][i]["mixer"], 1e-5), w[p + "norm1"], 1e-5)
        x = x + S.token_input(x, w["side.embed"][toks][:, 3 * i:3 * i + 3], w, p + "side.", 1e-5)
        assert np.abs(after[i] - x).max() < 1e-14
    assert np.abs(z - S.rms_norm(x, w["final.norm"], 1e-5) @ w["embed"].T).max() < 1e-14
