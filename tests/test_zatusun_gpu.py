"""Zatusun on the GPU, against the plain model in tests/plain_zatusun.py (numpy float64): every mechanism alone, then
whole models through the engine's step function, its scheduler, the trace runner and the command line.  Weights and
configurations are made here."""

import copy
import os
import tempfile

import numpy as np
import pytest
import torch

import plain_zatusun as S
import tiny_zatusun as tiny
from part_harness import DT, TOL, TOL_MODEL, _Manager, _ctx, _err, _make, _run_in_steps, _same, _w

pytestmark = pytest.mark.gpu

CUTS = [[(0, 8), (1, 1)], [(0, 9), (1, 1)], [(0, 2), (1, 30)], [(0, 1), (1, 1)], [(0, 44)], [(0, 1)], [(0, 1)], [(0, 4)]]


def _f32(a, dev="cuda"):
    return torch.as_tensor(np.asarray(a), dtype=torch.float32).to(dev).contiguous()


# --------------------------------------------------------------------------- embedding, norm, the start of a pass

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_embedding_takes_its_factor_and_the_positions_vector(dtype):
    from kv_cache_optimization_for_llm_b200.engine.batch import BatchBuilder, StepEntry
    rng = np.random.default_rng(0)
    ctx = _ctx(dtype)
    table, t64 = _w(rng, (31, 24), 0.5)
    pos, p64 = _w(rng, (20, 24), 0.5)
    emb = _make("embedding", "positioned_token_embedding", {"vocab_size": 31, "hidden_size": 24, "scale": 3.7, "positions": 20},
                {"table": table, "position_table": pos}, ctx)
    builder = BatchBuilder(64, 4, [8], ctx.device, ctx.status)
    toks = [rng.integers(0, 31, n).tolist() for n in (9, 1)]
    batch = builder.build([StepEntry(0, toks[0], 0, ()), StepEntry(1, toks[1], 19, ())],
                          _Manager({0: list(range(8)), 1: list(range(8))}, {0: 0, 1: 1}))
    x = emb.forward(batch).cpu().numpy()
    assert x.dtype == np.float32
    # single tokens come first in a step; float32 sums in both precisions
    ref = np.concatenate([t64[toks[1]] * 3.7 + p64[[19]], t64[toks[0]] * 3.7 + p64[:9]])
    assert np.abs(x - ref).max() < 1e-6
    # beyond the table: reported, nothing read
    batch = builder.build([StepEntry(0, toks[0], 12, ())], _Manager({0: list(range(8))}, {0: 0}))
    emb.forward(batch)
    assert int(ctx.status.item()) == 2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("W", [40, 7, 264])
def test_norm_with_a_weight_around_zero(dtype, W):
    rng = np.random.default_rng(1)
    ctx = _ctx(dtype)
    weight, w64 = _w(rng, (W,), 0.4)
    norm = _make("norm", "rmsnorm", {"size": W, "eps": 1e-3, "around_zero": True}, {"weight": weight}, ctx)
    x, x64 = _w(rng, (5, W), 0.1)            # small enough that eps, inside the root, shows
    d, d64 = _w(rng, (5, W), 0.1)
    xd = _f32(x64)
    got = norm.forward(xd, d.to(DT[dtype]).cuda())
    assert _err(got, S.centred_rms_norm(x64 + d64, w64, 1e-3), dtype) < (1e-6 if dtype == "float32" else 5e-3)
    assert np.abs(xd.cpu().numpy() - (x64 + d64)).max() < 1e-6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,W", [(5, 40), (130, 64), (3, 7)])
def test_a_pass_starts_from_a_product_over_stream_and_embedding(dtype, T, W):
    """The stream behind the next norm, and that norm's output, with and without a branch output still pending."""
    rng = np.random.default_rng(2)
    ctx = _ctx(dtype)
    w_in, in64 = _w(rng, (W, 2 * W), 0.2)
    steps, s64 = _w(rng, (3, W), 0.5)
    weight, w64 = _w(rng, (W,), 0.2)
    norm = _make("norm", "rmsnorm", {"size": W, "eps": 1e-5, "around_zero": True}, {"weight": weight}, ctx)
    parts = [_make("stream", "pass_entry", {"size": W, "passes": 3, "index": t}, {"in": w_in, "steps": steps}, ctx) for t in range(3)]
    (x, x64), (x0, e64), (d, d64) = (_w(rng, (T, W), 1.0) for _ in range(3))
    w = {"loop.in": in64, "loop.step": s64}
    made = parts[0].from_embedding(_f32(e64))
    for t, delta in ((0, None), (1, d.to(DT[dtype]).cuda()), (2, d.to(DT[dtype]).cuda())):
        stream = _f32(x64)
        h = norm.forward(stream, parts[t].forward(stream, delta, made))
        ref = S.start_pass(x64 + (0.0 if delta is None else d64), e64, w, t)
        tol = 2e-6 if dtype == "float32" else 6e-3
        assert np.abs(stream.cpu().numpy() - ref).max() < tol * np.abs(ref).max()
        assert _err(h, S.centred_rms_norm(ref, w64, 1e-5), dtype) < (5e-6 if dtype == "float32" else 1e-2)


# --------------------------------------------------------------------------- differential attention

def _att_params(H, m, eps=1e-5):
    from kv_cache_optimization_for_llm_b200.models.zatusun import _position
    return {"hidden_size": H, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"],
            "scale": m["scale"], "diff": m["diff"], "chunk": (m.get("mask") or {}).get("size"), "eps": eps,
            "position": _position(m, "attention")}


def _att_weights(rng, H, m):
    Hq, G, D, Dv = (m[k] for k in ("heads", "kv_heads", "dim", "vdim"))
    wt, w64 = {}, {}
    for n, shape, std in (("q", (Hq * 2 * D, H), 0.3), ("k", (G * 2 * D, H), 0.3), ("v", (G * Dv, H), 0.3), ("lq1", (D,), 0.3),
                          ("lk1", (D,), 0.3), ("lq2", (D,), 0.3), ("lk2", (D,), 0.3), ("o", (H, Hq * Dv), 0.3)):
        wt[n], w64[n] = _w(rng, shape, std)
    return wt, w64


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [
    dict(),
    dict(heads=3, kv_heads=1, dim=24, vdim=8, scale=0.2, diff=0.1, size=5, rot_dims=10, scaling=None),
    dict(heads=2, kv_heads=2, dim=8, vdim=40, scale=0.5, size=16, rot_dims=8),
    dict(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.125, diff=0.7, size=33, rot_dims=32),
    dict(heads=1, kv_heads=1, dim=5, vdim=3, scale=1.0, size=1, rot_dims=4),
    dict(heads=4, kv_heads=1, dim=32, vdim=64, scale=0.3, size=None, rot_dims=None),
    dict(heads=8, kv_heads=2, dim=40, vdim=32, scale=0.15, size=64, rot_dims=40),
    dict(heads=6, kv_heads=1, dim=128, vdim=128, scale=0.06, size=40, rot_dims=64),
    dict(heads=4, kv_heads=4, dim=64, vdim=128, scale=0.1, diff=0.8, size=None, rot_dims=2),
])
def test_attention_alone_in_portions_and_beside_another_request(dtype, shape):
    """Several shapes (grouped and ungrouped heads, key and value sizes that differ, blocks of one position, no blocks,
    no rotation, every channel turning), 70 and 33 tokens on pages of 8 that lie scattered; portions end inside pages
    and blocks and on their borders."""
    from kv_cache_optimization_for_llm_b200 import ops
    rng = np.random.default_rng(3)
    ctx = _ctx(dtype)
    H = 40
    m = tiny.attention(**shape)
    wt, w64 = _att_weights(rng, H, m)
    mixer = _make("mixer", "differential_chunk_attention", _att_params(H, m), wt, ctx)
    assert abs(mixer.lam - S.difference_weight(w64, "", m["diff"])) < 1e-12
    xs, refs = {}, {}
    for r, T in enumerate((70, 33)):
        x, x64 = _w(rng, (T, H), 1.0)
        xs[r], refs[r] = x.to(DT[dtype]).cuda(), S.attention_mixer(x64, w64, "", m, 1e-5)
    before = ops.choices["window_flash_attention_pair"]
    whole = _run_in_steps(mixer, ctx, xs, [[(0, 70)], [(1, 33)]])
    # bfloat16 prompt portions of sizes that are multiples of 8 run on tensor cores, everything else does not
    assert (ops.choices["window_flash_attention_pair"] > before) == (dtype == "bfloat16" and m["dim"] % 8 == 0 and m["vdim"] % 8 == 0)
    cut = _run_in_steps(mixer, ctx, xs, CUTS)
    one = _run_in_steps(mixer, ctx, {0: xs[1]}, [[(0, 1)]] * 33)
    for r in xs:
        assert _err(whole[r], refs[r], dtype) < TOL[dtype]
        assert _err(cut[r], refs[r], dtype) < TOL[dtype]
        assert _same(whole[r], cut[r], dtype), "a token's result must not depend on the cut or on the batch"
    assert _same(one[0], whole[1], dtype), "token by token"


def _spiked(dtype, chunk, T, query, spikes, lam=0.5, diff=0.3, page=8, D=16, Dv=None, flash=None):
    """The attention kernel alone on keys and values made so that one key a map decides: every query and key is small
    but the query at ``query`` and the keys in ``spikes`` (map -> key), whose raw scores are 30; the value of key j is
    the unit vector j mod Dv.  Returns what the query reads, in a prompt (one portion; ``flash``: the tile height of the
    tensor-core kernel, None: the general one) and decoded alone, and the plain answer."""
    from kv_cache_optimization_for_llm_b200 import ops
    from kv_cache_optimization_for_llm_b200.engine.batch import BatchBuilder, StepEntry
    ctx = _ctx(dtype)
    rng = np.random.default_rng(T + query)
    q, k = rng.normal(size=(2, T, 1, 2, D)) * 0.01
    for m, key in spikes.items():
        q[query, 0, m] = k[key, 0, m] = 0
        q[query, 0, m, 3], k[key, 0, m, 3] = 6.0, 5.0
    Dv = Dv or min(T, 128)
    v = np.zeros((T, 1, Dv))
    v[np.arange(T), 0, np.arange(T) % Dv] = 1.0
    ref = S.two_map_attention(q, k, v, 1.0, chunk or None, lam, diff, 1e-9)[query, 0]
    src = torch.as_tensor(np.concatenate([a.reshape(T, -1) for a in (q, k, v)], axis=1), dtype=torch.float32).to(DT[dtype]).cuda()
    outs = []
    for steps in ([T], [query] + [1] * (T - query)):
        pages = torch.zeros((T // page + 2, 1, page, 2 * D + Dv), dtype=DT[dtype], device="cuda")
        tables = {0: list(range(T // page + 1))[::-1]}
        builder = BatchBuilder(1024, 4, [64], ctx.device, ctx.status)
        at, rows = 0, []
        for n in [s for s in steps if s]:
            batch = builder.build([StepEntry(0, [0] * n, at, ())], _Manager(tables, {0: 0}))
            qq = ops.qk_rot_append(src[at:at + n].contiguous(), 0, 2 * D, 4 * D, None, None, None, None, None, 0.0, None, None, 0,
                                   "pairs", pages, batch.block_tables[0], batch, 1, 1, D, Dv, maps=2)
            got = ops.pair_attention(qq, pages, batch.block_tables[0], batch, 1, 1, D, Dv, 1.0, lam, 1e-9, 1.0 - diff,
                                     chunk=chunk, tensor_cores=flash is not None and n > 1, wide=flash)
            rows.append(got.float().cpu())
            at += n
        outs.append(torch.cat(rows)[query].numpy())
    assert int(ctx.status.item()) == 0
    return outs, ref


def _check_spikes(dtype, flash, tol):
    size, T, query = 37, 250, 245            # the query's block starts at 222
    for key, seen in ((222, True), (221, False), (0, False), (query, True), (224, True), (223, True), (query - 36, False),
                      (query - 37, False), (192, False), (191, False)):
        for m in (0, 1):
            (prompt, decoded), ref = _spiked(dtype, size, T, query, {m: key}, flash=flash)
            at, top = key % 128, np.abs(ref).max()
            assert (abs(ref[at]) > 0.9 * top) == seen      # the key stands out, or is not there at all
            if seen:
                assert np.sign(ref[at]) == (1 if m == 0 else -1)
            for got in (prompt, decoded):
                assert np.abs(got - ref).max() < tol * top, (key, m)
    for first, second in ((222, 230), (244, 223)):       # the maps pick different keys; each keeps its own sign
        outs, ref = _spiked(dtype, size, T, query, {0: first, 1: second}, flash=flash)
        assert ref[first % 128] > 0 > ref[second % 128] and all(np.abs(o - ref).max() < tol * np.abs(ref).max() for o in outs)
    outs, ref = _spiked(dtype, size, T, query, {0: 230, 1: 230}, lam=0.25, flash=flash)       # both pick the same one
    assert ref[230 % 128] > 0 and all(np.abs(o - ref).max() < tol * np.abs(ref).max() for o in outs)
    # the first position of a block sees only itself, the last one the block's first; blocks that are longer than the sequence
    for size_, T_, query_, key in ((37, 230, 222, 221), (37, 230, 221, 185), (64, 8, 2, 0)):
        outs, ref = _spiked(dtype, size_, T_, query_, {0: key}, flash=flash)
        assert all(np.abs(o - ref).max() < tol * np.abs(ref).max() for o in outs)
    for key in (2, 0, 63, 64, 127, 128):                 # no blocks: a key hundreds of tokens back, across all tiles
        outs, ref = _spiked(dtype, 0, 250, 249, {0: key}, flash=flash)
        assert ref[key % 128] > 0.9 * np.abs(ref).max() and all(np.abs(o - ref).max() < tol * np.abs(ref).max() for o in outs)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_keys_far_away_and_at_the_edges_of_a_block_in_either_map(dtype):
    _check_spikes(dtype, None, 1e-5 if dtype == "float32" else 2e-2)


@pytest.mark.parametrize("wide", [False, True])
def test_prompt_portions_on_tensor_cores_see_the_same_keys(wide):
    from kv_cache_optimization_for_llm_b200 import ops
    before = ops.choices["window_flash_attention_pair"]
    _check_spikes("bfloat16", wide, 2e-2)
    assert ops.choices["window_flash_attention_pair"] >= before + 30


# --------------------------------------------------------------------------- latent attention

def _lat_params(H, m, eps=1e-5):
    from kv_cache_optimization_for_llm_b200.models.zatusun import _position
    return {"hidden_size": H, **{k: m[k] for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale")}, "sink": False,
            "gate": True, "eps": eps, "position": _position(m, "latent_attention")}


def _lat_weights(rng, H, m):
    a, d, r, dv, qr, kr = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
    wt, w64 = {}, {}
    for role, name, shape, std, mean in (("dq", "dq", (qr, H), 0.3, 0), ("dq_norm", "dq.norm", (qr,), 0.2, 1.0),
                                         ("uq", "uq", (a * (d + r), qr), 0.3, 0), ("dkv", "dkv", (kr + r, H), 0.3, 0),
                                         ("dkv_norm", "dkv.norm", (kr,), 0.2, 1.0), ("uk", "uk", (a * d, kr), 0.3, 0),
                                         ("uv", "uv", (a * dv, kr), 0.3, 0), ("g", "g", (a * dv, H), 0.3, 0),
                                         ("o", "o", (H, a * dv), 0.3, 0)):
        wt[role], w64[name] = _w(rng, shape, std, mean)
    return wt, w64


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [dict(), dict(heads=1, dim=5, rot_dim=2, vdim=3, q_rank=6, kv_rank=4),
                                   dict(heads=9, dim=8, rot_dim=16, vdim=16, q_rank=24, kv_rank=64),
                                   dict(heads=2, dim=24, rot_dim=32, vdim=40, q_rank=16, kv_rank=96, scaling=None)])
def test_latent_attention_without_sink_with_gate_in_portions_and_beside_another_request(dtype, shape):
    from kv_cache_optimization_for_llm_b200 import ops
    rng = np.random.default_rng(5)
    ctx = _ctx(dtype)
    H = 40
    m = tiny.latent(**shape)
    wt, w64 = _lat_weights(rng, H, m)
    mixer = _make("mixer", "latent_attention", _lat_params(H, m), wt, ctx)
    xs, refs = {}, {}
    for r, T in enumerate((70, 33)):
        x, x64 = _w(rng, (T, H), 1.0)
        xs[r], refs[r] = x.to(DT[dtype]).cuda(), S.latent_attention_mixer(x64, w64, "", m, 1e-5)
    before = ops.choices["latent_attention_tc"]
    whole = _run_in_steps(mixer, ctx, xs, [[(0, 70)], [(1, 33)]])
    assert (ops.choices["latent_attention_tc"] > before) == (dtype == "bfloat16" and m["kv_rank"] % 16 == 0
                                                             and (m["kv_rank"] + m["rot_dim"]) % 16 == 0)
    cut = _run_in_steps(mixer, ctx, xs, CUTS)
    for r in xs:
        assert _err(whole[r], refs[r], dtype) < TOL[dtype]
        assert _err(cut[r], refs[r], dtype) < TOL[dtype]
        assert _same(whole[r], cut[r], dtype)
    # the gate shows: without it the plain answer is another one
    open_gate = S.latent_attention_mixer(xs[0].double().cpu().numpy(), dict(w64, g=np.zeros_like(w64["g"])), "", m, 1e-5)
    assert np.abs(open_gate - refs[0]).max() > 0.05 * np.abs(refs[0]).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kv_rank", [24, 32])
def test_latent_attention_finds_one_far_key(dtype, kv_rank):
    """300 tokens; the shared turned key part of token 5 is blown up so that its score stands out among hundreds (the
    slow waves of the rotation hardly turn it); the plain result changes by a large factor without that key."""
    rng = np.random.default_rng(11)
    ctx = _ctx(dtype)
    H, T = 40, 300
    m = tiny.latent(heads=2, dim=8, rot_dim=16, vdim=8, q_rank=12, kv_rank=kv_rank, base=1e6, scaling=dict(tiny.YARN, factor=8.0))
    wt, w64 = _lat_weights(rng, H, m)
    x, x64 = _w(rng, (T, H), 1.0)
    x[5] *= 16.0           # a power of two: bfloat16 holds the product exactly
    x64[5] *= 16.0
    ref = S.latent_attention_mixer(x64, w64, "", m, 1e-5)
    without = x64.copy()
    without[5] /= 16.0
    assert np.abs(ref[6:] - S.latent_attention_mixer(without, w64, "", m, 1e-5)[6:]).max() > 0.3 * np.abs(ref).max()
    mixer = _make("mixer", "latent_attention", _lat_params(H, m), wt, ctx)
    got = _run_in_steps(mixer, ctx, {0: x.to(DT[dtype]).cuda()}, [[(0, 3)], [(0, 5)], [(0, 120)], [(0, 1)], [(0, 127)], [(0, 2)]]
                        + [[(0, 1)]] * 42)
    assert _err(got[0], ref, dtype) < (3e-5 if dtype == "float32" else 0.08)


@pytest.mark.parametrize("T,H,N,K", [(130, 3, 24, 16), (200, 5, 7, 12), (4, 3, 24, 16)])
def test_per_head_products_with_a_gate(T, H, N, K):
    """bfloat16 steps of few rows (this package's kernel) and of many (the library's batched product, then one kernel
    that brings a token's heads together and applies the gate)."""
    from kv_cache_optimization_for_llm_b200 import ops
    rng = np.random.default_rng(6)
    x, x64 = _w(rng, (T, H * K + 8), 1.0)
    w, w64 = _w(rng, (H, N, K), 0.3)
    g, g64 = _w(rng, (T, 16 + H * N), 1.0)
    ref = np.einsum("hnk,thk->thn", w64, x64[:, 8:].reshape(T, H, K)).reshape(T, H * N)
    xc, wc, gc = (t.to(torch.bfloat16).cuda() for t in (x, w, g))
    assert _err(ops.head_gemm(xc, 8, K, wc), ref, "bfloat16") < 6e-3
    assert _err(ops.head_gemm(xc, 8, K, wc, (gc, 16)), ref * S.sigmoid(g64[:, 16:]), "bfloat16") < 6e-3


# --------------------------------------------------------------------------- linear attention with a decay per channel

def _lin_weights(rng, H, m, low=(0.0, 0.9), bias=1.0):
    a, n, dv = m["heads"], m["dim"], m["vdim"]
    wt, w64 = {}, {}
    for role, name, shape, std, mean in (("q", "q", (a * n, H), 0.3, 0), ("f", "f", (a * n, H), 0.3, 0), ("v", "v", (a * dv, H), 0.3, 0),
                                         ("f_bias", "f.b", (a * n,), 1.0, bias), ("norm", "norm", (dv,), 0.2, 1.0),
                                         ("o", "o", (H, a * dv), 0.3, 0)):
        wt[role], w64[name] = _w(rng, shape, std, mean)
    t = torch.as_tensor(rng.uniform(*low, size=(a * n,)), dtype=torch.float32).to(torch.bfloat16)
    wt["lower"], w64["lower"] = t, t.float().numpy().astype(np.float64)
    return wt, w64


def _lin_params(H, m, eps=1e-5):
    return {"hidden_size": H, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"], "eps": eps}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [dict(), dict(heads=1, dim=5, vdim=3), dict(heads=2, dim=16, vdim=16), dict(heads=2, dim=8, vdim=72),
                                   dict(heads=4, dim=64, vdim=32), dict(heads=1, dim=130, vdim=36), dict(heads=2, dim=12, vdim=136),
                                   dict(heads=1, dim=100, vdim=128), dict(heads=2, dim=48, vdim=18)])
def test_linear_attention_alone_in_portions_and_beside_another_request(dtype, shape):
    """Several shapes (one head, keys that are no multiple of four wide, heads whose norm runs in the scan and heads too
    wide for it), 70 and 33 tokens; the state slots start full of rubbish, which a request that starts at position 0
    must not read."""
    rng = np.random.default_rng(4)
    ctx = _ctx(dtype)
    H = 40
    m = tiny.hgrn2(**shape)
    wt, w64 = _lin_weights(rng, H, m)
    mixer = _make("mixer", "decayed_linear_attention", _lin_params(H, m), wt, ctx)
    xs, refs = {}, {}
    for r, T in enumerate((70, 33)):
        x, x64 = _w(rng, (T, H), 1.0)
        xs[r], refs[r] = x.to(DT[dtype]).cuda(), S.hgrn2_mixer(x64, w64, "", m, 1e-5)
    whole = _run_in_steps(mixer, ctx, xs, [[(0, 70)], [(1, 33)]])
    cut = _run_in_steps(mixer, ctx, xs, CUTS)
    one = _run_in_steps(mixer, ctx, {0: xs[1]}, [[(0, 1)]] * 33)
    tol = 1e-4 if dtype == "float32" else TOL[dtype]
    for r in xs:
        assert _err(whole[r], refs[r], dtype) < tol
        assert _err(cut[r], refs[r], dtype) < tol
        assert _same(whole[r], cut[r], dtype)
    assert _same(one[0], whole[1], dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [dict(heads=2, dim=12, vdim=20), dict(heads=1, dim=10, vdim=132), dict(heads=3, dim=32, vdim=64)])
def test_long_runs_are_walked_in_chunks_side_by_side_and_memories_last_for_hundreds_of_tokens(dtype, shape):
    """A run of 700 tokens (cut into chunks that are walked side by side) beside a short one, one of 1100, then 40
    tokens one by one; decays near one, so that the first tokens still show at the end."""
    from kv_cache_optimization_for_llm_b200 import ops
    rng = np.random.default_rng(6)
    ctx = _ctx(dtype, max_positions=2048)
    H = 24
    m = tiny.hgrn2(**shape)
    wt, w64 = _lin_weights(rng, H, m, low=(0.99, 0.9999))
    mixer = _make("mixer", "decayed_linear_attention", _lin_params(H, m), wt, ctx)
    xs, refs = {}, {}
    for r, T in enumerate((740, 90)):
        x, x64 = _w(rng, (T, H), 1.0)
        x64[:60] = np.abs(x64[:60])                         # the first tokens pull the memory one way
        x[:60] = x[:60].abs()
        xs[r], refs[r] = x.to(DT[dtype]).cuda(), S.hgrn2_mixer(x64, w64, "", m, 1e-5)
    before = ops.choices["linear_scan_chunked"]
    got = _run_in_steps(mixer, ctx, xs, [[(1, 5)], [(0, 700), (1, 1)], [(1, 84)]] + [[(0, 1)]] * 40, page=16, state_slots=4)
    assert ops.choices["linear_scan_chunked"] > before
    short = _run_in_steps(mixer, ctx, xs, [[(0, 200), (1, 90)], [(0, 255)], [(0, 245)]] + [[(0, 1)]] * 40, page=16, state_slots=4)
    tol = 3e-4 if dtype == "float32" else TOL[dtype]
    for r in xs:
        assert _err(got[r], refs[r], dtype) < tol and _err(short[r], refs[r], dtype) < tol
    late = S.hgrn2_mixer(xs[0][100:].double().cpu().numpy(), w64, "", m, 1e-5)
    assert np.abs(late[-1] - refs[0][-1]).max() > 1e-2 * np.abs(refs[0][-1]).max()


def test_a_run_of_more_than_a_thousand_tokens_from_a_state_and_beside_others():
    """float32, longer chunks: 1000 tokens, then 30, then a portion of 1024 that starts from a state, in one step with a
    run of two chunks and one of a single chunk."""
    rng = np.random.default_rng(8)
    ctx = _ctx("float32", max_positions=4096)
    H, m = 16, tiny.hgrn2(heads=2, dim=16, vdim=24)
    wt, w64 = _lin_weights(rng, H, m, low=(0.9, 0.999))
    mixer = _make("mixer", "decayed_linear_attention", _lin_params(H, m), wt, ctx)
    from kv_cache_optimization_for_llm_b200.cache.specs import SlotStateBinding
    from kv_cache_optimization_for_llm_b200.engine.batch import BatchBuilder, StepEntry
    lens = {0: 2054, 1: 200, 2: 90}
    xs = {r: _w(rng, (T, H), 1.0) for r, T in lens.items()}
    state = torch.full((4,) + mixer.cache_spec().shape, 3.0, device="cuda")
    builder = BatchBuilder(2048, 4, [300], ctx.device, ctx.status)
    manager = _Manager({r: list(range(300)) for r in lens}, {0: 2, 1: 0, 2: 1})
    at, got = dict.fromkeys(lens, 0), {r: [] for r in lens}
    for step in ([(0, 1000)], [(0, 30)], [(2, 90), (0, 1024), (1, 200)]):
        batch = builder.build([StepEntry(r, [0] * n, at[r], ()) for r, n in step], manager)
        y = mixer.forward(torch.cat([xs[r][0][at[r]:at[r] + n] for r, n in step]).float().cuda(), batch, SlotStateBinding(state=state))
        for (r, n), rows in zip(step, y.split([n for _, n in step])):
            got[r].append(rows.cpu())
            at[r] += n
    for r in lens:
        assert _err(torch.cat(got[r]), S.hgrn2_mixer(xs[r][1], w64, "", m, 1e-5), "float32") < 2e-4


# --------------------------------------------------------------------------- the experts

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [dict(), dict(experts=3, top=1, ff=16, limit=2.0), dict(experts=4, top=4, ff=8, limit=0.3),
                                   dict(experts=9, top=3, ff=5, limit=0.9), dict(experts=1, top=1, ff=24, limit=1.0)])
def test_experts_weigh_their_output_and_limit_both_products(dtype, shape):
    """Limits low enough that many features meet them, so that a weight on the input, a limit on the wrong side, or
    weights from a softmax over all experts would show."""
    rng = np.random.default_rng(7)
    ctx = _ctx(dtype)
    H, T = 40, 29
    mlp = tiny.moe(**shape)
    E, F, top = mlp["router"]["experts"], mlp["expert"]["ff"], mlp["router"]["top"]
    wt, w64 = {}, {}
    wt["router"], w64["router"] = _w(rng, (E, H), 0.5)
    for e in range(E):
        for role, shp in (("gate", (F, H)), ("up", (F, H)), ("down", (H, F))):
            wt[f"{role}{e}"], w64[f"e{e}.{role}"] = _w(rng, shp, 0.3)
    params = {"hidden_size": H, "experts": E, "top": top, "expert_ff": F, "limit": mlp["expert"]["limit"], "shared_ff": 0,
              "alpha": 1.702, "score": "softmax_chosen", "weigh": "output"}
    ff = _make("feed_forward", "limited_experts", params, wt, ctx)
    x, x64 = _w(rng, (T, H), 1.0)
    ref = S.moe(x64, w64, "", mlp)
    assert _err(ff.forward(x.to(DT[dtype]).cuda(), None), ref, dtype) < TOL[dtype]
    chosen, weight = S.route(x64, w64["router"], top)
    wrong = np.zeros_like(ref)
    for t in range(T):
        for e, c in zip(chosen[t], weight[t]):
            wrong[t] += S.limited_expert((c * x64[t])[None], w64[f"e{e}.gate"], w64[f"e{e}.up"], w64[f"e{e}.down"],
                                         mlp["expert"]["limit"])[0]
    assert top == 1 or np.sqrt(((wrong - ref) ** 2).mean()) > 0.05 * np.sqrt((ref ** 2).mean())


def test_router_weights_are_a_softmax_over_the_chosen_logits():
    from kv_cache_optimization_for_llm_b200 import ops
    z = np.array([[2.0, -1.0, 0.5, 3.0, -4.0], [0.1, 0.2, 0.3, -0.1, 0.0], [-95.0, -6.0, -7.0, -8.0, -9.0], [60.0, 1.0, 59.0, -60.0, 2.0]])
    x = torch.zeros((4, 8), dtype=torch.float32, device="cuda")
    gate, _ = ops.route(x, None, None, 5, 0, 3, 1.0, _f32(z), score="softmax", renormalize=True)
    chosen, weight = S.route(z, np.eye(5), 3)
    ref = np.zeros((4, 5))
    np.put_along_axis(ref, chosen, weight, axis=1)
    assert np.abs(gate.cpu().numpy() - ref).max() < 1e-6


# --------------------------------------------------------------------------- whole models

def _runner(folder, dtype, **kw):
    from kv_cache_optimization_for_llm_b200 import EngineConfig
    from kv_cache_optimization_for_llm_b200.engine.runner import ModelRunner
    args = dict(dtype=dtype, page_size=8, num_pages=40, max_num_seqs=3, max_num_batched_tokens=256, max_model_len=160,
                use_cuda_graphs=False)
    args.update(kw)
    return ModelRunner(folder, EngineConfig(**args))


def _logit_err(got, ref, dtype="float32"):
    """float32: the largest difference over the largest value.  bfloat16: root mean square of the differences over
    that of the values, row by row, and of the rows' figures the one that four in five stay below: where two experts'
    logits lie within a rounding of each other the choice may go either way, which changes a few rows much and says
    nothing about the kernels; all rows together must still stay below three times the limit."""
    if dtype == "float32":
        return np.abs(got - ref).max() / np.abs(ref).max()
    rows = np.sqrt(((got - ref) ** 2).mean(axis=-1)) / np.sqrt((ref ** 2).mean())
    if rows.ndim == 0 or rows.size < 5:
        return float(np.max(rows))
    return max(float(np.quantile(rows, 0.8)), float(np.sqrt((rows ** 2).mean())) / 3.0)


def _close(a, b, dtype):
    """Two runs of the engine that cut the same tokens differently."""
    return _logit_err(a, b, dtype) < (5e-5 if dtype == "float32" else TOL_MODEL[dtype])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_model_prefill_decoding_portions_batches_and_reuse(dtype):
    """A model with all kinds of mixer, layers without feed-forward and a repeated run of layers.  Whole prompts; token
    by token; portions of 2, 3, 7, ... beside single tokens of another request; then requests that end and others that
    take over their slots and pages in a pool that holds two of them at most; 60 decoded tokens in a row, past every
    block's end."""
    from kv_cache_optimization_for_llm_b200.engine.batch import StepEntry
    folder = tempfile.mkdtemp(prefix="kvb200_zs_")
    cfg = tiny.MIXED
    w = tiny.write_model(folder, cfg, seed=1)
    r = _runner(folder, dtype)
    assert len(r.spec.schedule) == 9 and len(r.spec.layers) == 6
    assert len(r.cache.states) == 3        # one linear attention in front of the repeated run, one in each of its passes
    rng = np.random.default_rng(5)
    seqs = [rng.integers(0, cfg["vocab"], n).tolist() for n in (90, 37, 61, 1, 150)]
    refs = [S.forward(cfg, w, s) for s in seqs]
    tol = TOL_MODEL[dtype]
    whole = r.step([StepEntry(0, seqs[1], 0, range(37))]).cpu().numpy()
    assert _logit_err(whole, refs[1], dtype) < tol
    r.release(0)
    single = np.concatenate([r.step([StepEntry(1, [t], i, [0])]).cpu().numpy() for i, t in enumerate(seqs[1])])
    assert _logit_err(single, refs[1], dtype) < tol
    assert _close(whole, single, dtype)
    r.release(1)
    got2 = [r.step([StepEntry(12, seqs[2][:20], 0, range(20))]).cpu().numpy()]
    pos0, pos2, got0 = 0, 20, []
    for n in (2, 3, 7, 1, 8, 16, 2, 9, 5, 1, 1, 30, 2, 3):
        entries = [StepEntry(10, seqs[0][pos0:pos0 + n], pos0, range(n))]
        if pos2 < len(seqs[2]):
            entries.insert(0 if n % 2 else 1, StepEntry(12, [seqs[2][pos2]], pos2, [0]))
        if n == 7:
            entries.append(StepEntry(13, seqs[3], 0, [0]))
        out = r.step(entries).cpu().numpy()
        i = 0
        for e in entries:
            k = len(e.want)
            if e.request_id == 10:
                got0.append(out[i:i + k])
            elif e.request_id == 12:
                got2.append(out[i:i + k])
                pos2 += 1
            else:
                assert _logit_err(out[i:i + k], refs[3], dtype) < tol
                r.release(13)
            i += k
        pos0 += n
    assert pos0 == 90
    assert _logit_err(np.concatenate(got0), refs[0], dtype) < tol
    assert _logit_err(np.concatenate(got2), refs[2][:pos2], dtype) < tol
    r.check_status()
    r.release(10)
    r.release(12)
    assert r.manager.check() == ""
    long = [r.step([StepEntry(20, seqs[4][:90], 0, range(90))]).cpu().numpy()]
    for i in range(90, 150):
        long.append(r.step([StepEntry(20, [seqs[4][i]], i, [0])]).cpu().numpy())
    assert _logit_err(np.concatenate(long), refs[4], dtype) < tol
    r.check_status()
    r.release(20)
    assert all(r.manager.free_pages(g) == 40 for g in range(r.manager.num_groups()))


def test_the_stream_after_every_layer():
    """float32: the residual stream after each run of a layer, against the plain model's; the wrong layouts of a pass's
    start (the embedding's output first, the vector ahead of the product) are far away."""
    from kv_cache_optimization_for_llm_b200 import ops
    from kv_cache_optimization_for_llm_b200.engine.batch import StepEntry
    folder = tempfile.mkdtemp(prefix="kvb200_zs_")
    cfg = tiny.MIXED
    w = tiny.write_model(folder, cfg, seed=3)
    r = _runner(folder, "float32")
    seq = np.random.default_rng(2).integers(0, cfg["vocab"], 30).tolist()
    _, after = S.forward(cfg, w, seq, keep_layers=True)
    seen = []
    for block in r.model.layers:
        inner = block.forward

        def spy(residual, delta, batch, cache, inner=inner):
            residual, pending = inner(residual, delta, batch, cache)
            copy_ = residual.clone()
            ops.add_norm(copy_, pending, None, None, 0.0, torch.float32)       # what is pending joins a copy of the stream
            seen.append(copy_.cpu().numpy())
            return residual, pending
        block.forward = spy
    r.step([StepEntry(0, seq, 0, [29])])
    assert len(seen) == len(after) == 9
    for i, (got, ref) in enumerate(zip(seen, after)):
        assert np.abs(got - ref).max() < 2e-5 * np.abs(ref).max(), f"after layer run {i}"
    swapped = dict(w, **{"loop.in": np.roll(w["loop.in"], 40, axis=1)})
    assert np.abs(S.forward(cfg, swapped, seq, keep_layers=True)[1][1] - after[1]).max() > 0.1 * np.abs(after[1]).max()


ODD = dict(heads=3, dim=5, vdim=7)


@pytest.mark.parametrize("layers,width,kw", [
    # one layer of each kind alone
    ([tiny.layer("hgrn2", tiny.hgrn2(heads=2, dim=8, vdim=8), tiny.moe(experts=2, top=1, ff=8))], 32, {}),
    ([tiny.layer("attention", tiny.attention(heads=2, kv_heads=1, dim=8, vdim=8, size=6, rot_dims=8))], 32, {}),
    ([tiny.layer("latent_attention", tiny.latent(heads=2, dim=8, rot_dim=8, vdim=8, q_rank=8, kv_rank=8),
                 tiny.moe(experts=4, top=4, ff=8))], 32, {}),
    # where the numbers that could be equal are not, constants that are 1 or absent, no blocks, a run of one layer three times
    ([tiny.layer("latent_attention", tiny.latent(heads=6, dim=24, rot_dim=40, vdim=56, q_rank=72, kv_rank=88, scale=0.11),
                 tiny.moe(experts=7, top=3, ff=24, limit=0.5)),
      tiny.layer("attention", tiny.attention(heads=6, kv_heads=3, dim=24, vdim=40, scale=0.15, size=None, rot_dims=24, base=77.0)),
      tiny.layer("hgrn2", tiny.hgrn2(heads=5, dim=20, vdim=12)),
      tiny.layer("attention", tiny.attention(heads=1, kv_heads=1, dim=96, vdim=16, scale=0.05, size=64, rot_dims=None),
                 tiny.moe(experts=2, top=2, ff=104)),
      tiny.layer("hgrn2", tiny.hgrn2(heads=1, dim=4, vdim=100), tiny.moe())], 104,
     dict(emb_scale=1.0, logit_softcap=None, loop=(1, 2, 3))),
    # sizes that are no multiples of eight: nothing may rest on 16-byte rows; the repeated run ends the model
    ([tiny.layer("attention", tiny.attention(heads=3, kv_heads=1, dim=5, vdim=3, scale=0.4, size=7, rot_dims=2),
                 tiny.moe(experts=3, top=2, ff=9)),
      tiny.layer("hgrn2", tiny.hgrn2(**ODD), tiny.moe(experts=2, top=1, ff=3)),
      tiny.layer("latent_attention", tiny.latent(heads=2, dim=6, rot_dim=6, vdim=9, q_rank=5, kv_rank=10))], 36,
     dict(logit_softcap=0.5, loop=(1, 3, 2))),
    # a width that is no multiple of four; every layer in a run that goes through once
    ([tiny.layer("hgrn2", tiny.hgrn2(), tiny.moe()), tiny.layer("attention", tiny.attention())], 27, dict(loop=(0, 2, 1))),
])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_other_orders_of_layers_sizes_and_constants(layers, width, kw, dtype):
    """A prompt in three portions and four tokens one by one, against the plain model."""
    from kv_cache_optimization_for_llm_b200.engine.batch import StepEntry
    folder = tempfile.mkdtemp(prefix="kvb200_zs_")
    cfg = tiny.config(layers, width=width, vocab=53, eps=1e-4, **kw)
    w = tiny.write_model(folder, cfg, seed=7)
    r = _runner(folder, dtype)
    seq = np.random.default_rng(1).integers(0, 53, 44).tolist()
    ref = S.forward(cfg, w, seq)
    got, pos = [], 0
    for n in (11, 2, 27, 1, 1, 1, 1):
        got.append(r.step([StepEntry(0, seq[pos:pos + n], pos, range(n))]).cpu().numpy())
        pos += n
    assert _logit_err(np.concatenate(got), ref, dtype) < TOL_MODEL[dtype]
    r.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_prompt_of_hundreds_of_tokens_at_once_and_in_portions(dtype):
    """400 tokens in one step (long bfloat16 products by the library, chunked scans, wide tiles) against portions, and
    both against the plain model."""
    from kv_cache_optimization_for_llm_b200.engine.batch import StepEntry
    folder = tempfile.mkdtemp(prefix="kvb200_zs_")
    cfg = copy.deepcopy(tiny.MIXED)
    cfg["max_positions"] = 512
    w = tiny.write_model(folder, cfg, seed=11)
    r = _runner(folder, dtype, num_pages=120, max_num_batched_tokens=512, max_model_len=480)
    seq = np.random.default_rng(3).integers(0, cfg["vocab"], 410).tolist()
    ref = S.forward(cfg, w, seq)
    runs = []
    for rid, cuts in enumerate(([400] + [1] * 10, [150, 2, 98, 130, 30])):
        pos, got = 0, []
        for n in cuts:
            got.append(r.step([StepEntry(rid, seq[pos:pos + n], pos, range(n))]).cpu().numpy())
            pos += n
        assert pos == 410
        runs.append(np.concatenate(got))
        assert _logit_err(runs[-1], ref, dtype) < (2e-4 if dtype == "float32" else TOL_MODEL[dtype])
        r.release(rid)
    assert _logit_err(runs[0], runs[1], dtype) < (2e-4 if dtype == "float32" else TOL_MODEL[dtype])
    r.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["mixed", "attention_only"])
def test_greedy_generation_through_the_engine_and_its_scheduler(dtype, which):
    """Prompts of unequal length through ``LLM.generate``: the scheduler's portions (a token budget of 24 per step),
    decode steps replayed from CUDA graphs, the engine one step ahead, five requests in three seats.  Every sampled
    row's logits are compared with the plain model on the final sequences, and in float32 the greedy tokens themselves.
    The model without a memory has no state of fixed size, so that its lone prompt portions and its steps of single
    tokens beside one portion are replayed from graphs too (with dummy tokens behind the run)."""
    from kv_cache_optimization_for_llm_b200 import LLM, SamplingParams
    from logit_hook import LogitRecorder
    folder = tempfile.mkdtemp(prefix="kvb200_zs_")
    cfg = tiny.MIXED if which == "mixed" else tiny.ATTENTION_ONLY
    w = tiny.write_model(folder, cfg, seed=4)
    llm = LLM(folder, dtype=dtype, page_size=8, num_pages=48, max_num_seqs=3, max_num_batched_tokens=24,
              max_model_len=128, use_cuda_graphs=True, run_ahead=True)
    rec = LogitRecorder(llm.engine.runner)
    rng = np.random.default_rng(9)
    prompts = [rng.integers(0, cfg["vocab"], n).tolist() for n in (3, 41, 17, 1, 30)]
    outs = llm.generate(prompts, SamplingParams(max_tokens=12, temperature=0.0, ignore_eos=True))
    assert [len(o) for o in outs] == [12] * 5
    seqs = {i: prompts[i] + outs[i] for i in range(5)}
    plain = {i: S.forward(cfg, w, seqs[i]) for i in seqs}
    if dtype == "float32":
        n, worst = rec.compare(seqs, lambda i: plain[i], TOL_MODEL[dtype], "greedy generation")
    else:       # the measure of this file's other bfloat16 comparisons: over all of a request's rows at once
        got = rec.collect(seqs)
        n = sum(len(ps) for ps, _ in got.values())
        for i, (ps, rows) in got.items():
            assert _logit_err(rows, plain[i][ps], dtype) < TOL_MODEL[dtype], f"greedy generation: request {i}"
    assert n >= 60 and llm.engine.runner._graphs
    if dtype == "float32":
        for i in seqs:
            for j, tok in enumerate(outs[i]):
                row = plain[i][len(prompts[i]) + j - 1]
                assert row[tok] >= row.max() - 1e-4 * np.abs(row).max(), (i, j)
    assert llm.engine.runner.manager.check() == ""


@pytest.mark.parametrize("dtype,flags", [("float32", ()), ("bfloat16", ()), ("float32", ("--cuda-graphs",))])
def test_replay_through_the_trace_runner(dtype, flags):
    """bin/trace_run on a Zatusun folder: each request whole, then four live requests whose portions (down to two
    tokens) run beside single tokens in a pool that holds exactly them, in four state slots; requests that end hand
    pages and slots to the ones that follow."""
    from trace_driver import TraceRun, ceil64
    folder = tempfile.mkdtemp(prefix="kvb200_zs_")
    cfg = tiny.MIXED
    w = tiny.write_model(folder, cfg, seed=9)
    rng = np.random.default_rng(2)
    seqs = [rng.integers(0, cfg["vocab"], n).tolist() for n in (70, 33, 50, 21)]
    refs = [S.forward(cfg, w, s) for s in seqs]
    tol = TOL_MODEL[dtype]
    tr = TraceRun(folder, dtype, sum(ceil64(len(s)) for s in seqs), ("--page-size", "8") + tuple(flags))
    try:
        for r, s in enumerate(seqs):
            got = tr.step([(f"w{r}", s, range(len(s)))], end=[f"w{r}"])
            assert _logit_err(got, refs[r], dtype) < tol, f"whole request {r}"
        for round_ in range(2):         # the second time in slots and pages that the first gave back
            plans = {0: [5, 2, 16, 9, 2, 30] + [1] * 6, 1: [1, 1, 20, 2] + [1] * 9, 2: [33, 2, 3, 2] + [1] * 10,
                     3: [2, 2, 2, 7] + [1] * 8}
            pos = {r: 0 for r in plans}
            step = 0
            while plans:
                entries, expect, ends = [], [], []
                for r in sorted(plans):
                    if step < r:        # they start one step apart
                        continue
                    n = plans[r].pop(0)
                    entries.append((f"m{round_}_{r}", seqs[r][pos[r]:pos[r] + n], range(n)))
                    expect.append(refs[r][pos[r]:pos[r] + n])
                    pos[r] += n
                    if not plans[r]:
                        assert pos[r] == len(seqs[r])
                        ends.append(f"m{round_}_{r}")
                        del plans[r]
                got = tr.step(entries, end=ends)
                assert _logit_err(got, np.concatenate(expect), dtype) < tol, f"time {round_}, mixed step {step}"
                step += 1
    finally:
        tr.close()


def test_command_line_serves_the_design():
    """The engine's command line on a Zatusun folder: requests on standard input in the wire format, greedy tokens
    back as JSON lines; each token is the plain model's best (ties within 1e-4 allowed)."""
    import json
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    folder = tempfile.mkdtemp(prefix="kvb200_zs_")
    cfg = tiny.MIXED
    w = tiny.write_model(folder, cfg, seed=8)
    rng = np.random.default_rng(4)
    prompts = {3: rng.integers(0, cfg["vocab"], 9).tolist(), 11: rng.integers(0, cfg["vocab"], 26).tolist()}
    lines = [f"{rid} 6 1 " + " ".join(map(str, toks)) for rid, toks in prompts.items()]
    env = dict(os.environ, IGNORE_EOS="1", PYTHONPATH=root + os.pathsep + os.environ.get("PYTHONPATH", ""))
    p = subprocess.run([sys.executable, "-m", "kv_cache_optimization_for_llm_b200.cli", folder, "--dtype", "float32",
                        "--page-size", "4", "--num-pages", "64", "--max-num-seqs", "4", "--max-model-len", "64"],
                       input="\n".join(lines) + "\n", capture_output=True, text=True, env=env, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    out = [json.loads(line) for line in p.stdout.splitlines() if line.strip()]
    for rid, prompt in prompts.items():
        toks = [m["tok"] for m in out if m.get("id") == rid and "tok" in m]
        assert len(toks) == 6
        logits = S.forward(cfg, w, prompt + toks)
        for j, tok in enumerate(toks):
            row = logits[len(prompt) + j - 1]
            assert row[tok] >= row.max() - 1e-4 * np.abs(row).max(), (rid, j)
