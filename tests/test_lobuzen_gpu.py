"""Lobuzen on the GPU, against the plain model in tests/plain_lobuzen.py (numpy float64): every mechanism alone, then
whole models through the engine's step function, its scheduler, the trace runner and the command line.  Weights and
configurations are made here."""

import os
import tempfile

import numpy as np
import pytest
import torch

import plain_lobuzen as S
import tiny_lobuzen as tiny
from part_harness import DT, TOL, TOL_MODEL, _Manager, _ctx, _err, _make, _run_in_steps, _same, _w

pytestmark = pytest.mark.gpu

CUTS = [[(0, 8), (1, 1)], [(0, 9), (1, 1)], [(0, 2), (1, 30)], [(0, 1), (1, 1)], [(0, 44)], [(0, 1)], [(0, 1)], [(0, 4)]]


def _f32(a, dev="cuda"):
    return torch.as_tensor(np.asarray(a), dtype=torch.float32).to(dev).contiguous()


def _mixer_against_plain(mixer, ctx, dtype, rng, H, plain, kernels=None):
    """70 and 33 tokens through a mixer alone: whole, in portions beside each other that end inside pages and windows and
    on their borders, and token by token."""
    from kv_cache_optimization_for_llm_b200 import ops
    xs, refs = {}, {}
    for r, T in enumerate((70, 33)):
        x, x64 = _w(rng, (T, H), 1.0)
        xs[r], refs[r] = x.to(DT[dtype]).cuda(), plain(x64)
    before = dict(ops.choices)
    whole = _run_in_steps(mixer, ctx, xs, [[(0, 70)], [(1, 33)]])
    for name, used in (kernels or {}).items():
        assert (ops.choices[name] > before.get(name, 0)) == used, name
    cut = _run_in_steps(mixer, ctx, xs, CUTS)
    one = _run_in_steps(mixer, ctx, {0: xs[1]}, [[(0, 1)]] * 33)
    for r in xs:
        assert _err(whole[r], refs[r], dtype) < TOL[dtype]
        assert _err(cut[r], refs[r], dtype) < TOL[dtype]
        assert _same(whole[r], cut[r], dtype), "a token's result must not depend on the cut or on the batch"
    assert _same(one[0], whole[1], dtype), "token by token"


# --------------------------------------------------------------------------- attention with unweighted norms

def _att_params(H, m, eps=1e-5):
    return {"hidden_size": H, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"],
            "scale": m["scale"], "window": S.window_size(m), "qk_norm": "unweighted", "eps": eps}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [
    dict(), dict(heads=3, kv_heads=1, dim=24, vdim=8, scale=0.5, size=5), dict(heads=2, kv_heads=2, dim=8, vdim=40, scale=1.0, size=16),
    dict(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.2, size=33), dict(heads=1, kv_heads=1, dim=5, vdim=3, scale=1.0, size=1),
    dict(heads=4, kv_heads=1, dim=32, vdim=64, scale=0.3, size=None), dict(heads=12, kv_heads=2, dim=128, vdim=128, scale=0.1, size=40),
    dict(heads=4, kv_heads=4, dim=64, vdim=128, scale=0.1, size=64), dict(heads=2, kv_heads=1, dim=72, vdim=136, scale=0.1, size=9),
])
def test_attention_alone_in_portions_and_beside_another_request(dtype, shape):
    rng = np.random.default_rng(3)
    ctx, H = _ctx(dtype), 40
    m = tiny.attention(**shape)
    Hq, G, D, Dv = (m[k] for k in ("heads", "kv_heads", "dim", "vdim"))
    wt, w64 = {}, {}
    for n, s in (("q", (Hq * D, H)), ("k", (G * D, H)), ("v", (G * Dv, H)), ("o", (H, Hq * Dv))):
        wt[n], w64[n] = _w(rng, s, 0.3)
    eps = 0.3                               # large enough that it, inside the root, shows
    mixer = _make("mixer", "shaped_window_attention", _att_params(H, m, eps), wt, ctx)
    tensor_cores = dtype == "bfloat16" and D % 8 == 0 and Dv % 8 == 0 and max(D, Dv) <= 128
    _mixer_against_plain(mixer, ctx, dtype, rng, H, lambda x: S.attention_mixer(x, w64, "", m, eps),
                         {"window_flash_attention": tensor_cores})


def _spiked_attention(dtype, window, T, query, key, dim, kernel):
    """The attention kernels alone (no norm in front) on keys made so that one decides: every query and key is small but
    the query at ``query`` and the key at ``key``, whose raw score is 30; key j's value is the unit vector j mod dim.  What
    the query reads in a prompt and decoded alone, and the plain answer."""
    from kv_cache_optimization_for_llm_b200 import ops
    from kv_cache_optimization_for_llm_b200.engine.batch import BatchBuilder, StepEntry
    ctx = _ctx(dtype)
    rng = np.random.default_rng(T + query)
    q, k = rng.normal(size=(2, T, 1, dim)) * 0.01
    q[query, 0] = k[key, 0] = 0
    q[query, 0, 3], k[key, 0, 3] = 6.0, 5.0
    v = np.zeros((T, 1, dim))
    v[np.arange(T), 0, np.arange(T) % dim] = 1.0
    ref = S.attend(q, k, v, 1.0, window)[query, 0]
    src = torch.as_tensor(np.concatenate([a.reshape(T, -1) for a in (q, k, v)], axis=1), dtype=torch.float32).to(DT[dtype]).cuda()
    page, outs = 8, []
    for steps in ([T], [query] + [1] * (T - query)):
        pages = torch.zeros((T // page + 2, 1, page, 2 * dim), dtype=DT[dtype], device="cuda")
        builder = BatchBuilder(1024, 4, [64], ctx.device, ctx.status)
        at, rows = 0, []
        for n in [s for s in steps if s]:
            # pages behind the window are gone, as the cache manager takes them back
            table = list(range(T // page + 1))[::-1]
            first = max(0, at - window + 1) // page if window else 0
            table[:first] = [-1] * first
            batch = builder.build([StepEntry(0, [0] * n, at, ())], _Manager({0: table}, {0: 0}))
            bt, rows_in = batch.block_tables[0], src[at:at + n].contiguous()
            qq = ops.qk_norm_append(rows_in, 0, dim, 2 * dim, None, None, None, None, None, 0.0, pages, bt, batch, 1, 1, dim, dim)
            if n == 1 or kernel is None:
                got = ops.window_attention(qq, 0, pages, bt, batch, 1, 1, dim, dim, 1.0, window or 0, 0, False)
            elif kernel == "roles":
                got = ops.flash_attention_rows(qq, pages, bt, batch, 1, 1, dim, 1.0, window or 0, 0, False, wide=3)
            else:
                got = ops.window_flash_attention(qq, pages, bt, batch, 1, 1, dim, dim, 1.0, window or 0, 0, False, wide=kernel == "wide")
            rows.append(got.float().cpu())
            at += n
        outs.append(torch.cat(rows)[query].numpy())
    assert int(ctx.status.item()) == 0
    return outs, ref


@pytest.mark.parametrize("dtype,kernel", [("float32", None), ("bfloat16", None), ("bfloat16", "narrow"), ("bfloat16", "wide"),
                                          ("bfloat16", "roles")])
def test_keys_far_away_and_at_the_edges_of_a_window(dtype, kernel):
    T, query = 250, 245
    for window, keys in ((37, ((209, True), (208, False), (245, True), (244, True), (216, True), (215, True), (0, False), (128, False))),
                         (1, ((245, True), (244, False))), (54, ((192, True), (191, False))), (118, ((128, True), (127, False))),
                         (246, ((0, True), (63, True))), (245, ((0, False), (1, True))), (None, ((0, True), (2, True), (127, True)))):
        for key, seen in keys:
            outs, ref = _spiked_attention(dtype, window, T, query, key, 64, kernel)
            assert (ref[key % 64] > 0.9) == seen or window == 1        # the key stands out, or is not there
            for got in outs:
                assert np.abs(got - ref).max() < (1e-5 if dtype == "float32" else 2e-2), (window, key)


# --------------------------------------------------------------------------- latent attention over a window, with a sink

def _lat_params(H, m, eps=1e-5, borrows=False):
    return {"hidden_size": H, **{k: m[k] for k in ("heads", "dim", "vdim", "kv_rank", "scale")}, "rot_dim": 0, "q_rank": None,
            "window": S.window_size(m), "sink": True, "borrows_latent": borrows, "split_decode": True, "eps": eps}


def _lat_weights(rng, H, m, borrows=False):
    a, d, dv, kr = (m[k] for k in ("heads", "dim", "vdim", "kv_rank"))
    wt, w64 = {}, {}
    for role, name, shape, std, mean in (("q", "q", (a * d, H), 0.3, 0), ("dkv", "dkv", (kr, H), 0.3, 0), ("dkv_norm", "dkv.norm", (kr,), 0.2, 1.0),
                                         ("uk", "uk", (a * d, kr), 0.3, 0), ("uv", "uv", (a * dv, kr), 0.3, 0), ("sink", "sink", (a,), 1.0, 2.0),
                                         ("o", "o", (H, a * dv), 0.3, 0)):
        if not (borrows and role.startswith("dkv")):
            wt[role], w64[name] = _w(rng, shape, std, mean)
    return wt, w64


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [
    dict(), dict(heads=1, dim=5, vdim=3, kv_rank=7, size=1), dict(heads=9, dim=8, vdim=16, kv_rank=64, size=33),
    dict(heads=2, dim=24, vdim=40, kv_rank=96, size=8), dict(heads=3, dim=16, vdim=8, kv_rank=48, size=40),
    dict(heads=70, dim=4, vdim=4, kv_rank=16, size=21), dict(heads=4, dim=32, vdim=24, kv_rank=80, size=None),
    dict(heads=2, dim=16, vdim=16, kv_rank=25, size=12), dict(heads=16, dim=16, vdim=16, kv_rank=512, scale=0.05, size=50),
    dict(heads=8, dim=12, vdim=20, kv_rank=160, scale=0.1, size=64),
])
def test_latent_attention_alone_in_portions_and_beside_another_request(dtype, shape):
    """Several shapes: latents that fill whole tiles of the tensor-core kernel and ones that do not (an odd one too), more
    heads than a tile has rows, windows of one token, of a page, and none."""
    rng = np.random.default_rng(5)
    ctx, H = _ctx(dtype), 40
    m = tiny.latent(**shape)
    wt, w64 = _lat_weights(rng, H, m)
    eps = 0.2
    mixer = _make("mixer", "latent_attention", _lat_params(H, m, eps), wt, ctx)
    plain = lambda x: S.latent_attention_mixer(x, S.latent(x, w64, "", eps), w64, "", m)
    from kv_cache_optimization_for_llm_b200 import ops
    on_tensor_cores = dtype == "bfloat16" and m["kv_rank"] % 16 == 0
    before = ops.choices["latent_decode"]
    _mixer_against_plain(mixer, ctx, dtype, rng, H, plain, {"latent_attention_tc": on_tensor_cores})
    assert (ops.choices["latent_decode"] > before) == on_tensor_cores
    # the sinks show: without them the plain answer is another one
    x = rng.normal(size=(40, H))
    bare = S.latent_attention_mixer(x, S.latent(x, w64, "", eps), dict(w64, sink=w64["sink"] - 1e9), "", m)
    assert np.abs(bare - plain(x)).max() > 0.02 * np.abs(plain(x)).max()


def _spiked_latents(dtype, window, T, query, key, rank, heads, sink, made=None):
    """The kernel alone: cached row j holds the unit vector 1 + j mod (rank - 1), the row at ``key`` also a 5 in channel 0,
    which only the query at ``query`` looks for, so that their score is 30 among zeros.  What every head of the query reads
    in a prompt (one portion) and decoded alone, and the plain answer.  ``made``: runs attend to keys and values made for the
    step (from matrices that hand the latent through), by the tcgen05 kernel ("roles") or with tiles of 64 or 128 rows."""
    from kv_cache_optimization_for_llm_b200 import ops
    from kv_cache_optimization_for_llm_b200.engine.batch import BatchBuilder, StepEntry
    ctx, page = _ctx(dtype), 8
    c = np.zeros((T, rank))
    c[np.arange(T), 1 + np.arange(T) % (rank - 1)] = 1.0
    c[key, 0] = 5.0
    q = np.zeros((T, heads, rank))
    q[query, :, 0] = 6.0
    sinks = np.full(heads, sink) + np.arange(heads) * 0.5
    ref = S.attend(q, np.repeat(c[:, None], heads, 1), np.repeat(c[:, None], heads, 1), 1.0, window, sinks)[query]
    pages = torch.zeros((T // page + 2, 1, page, rank), dtype=DT[dtype], device="cuda")
    order = list(range(T // page + 1))[::-1]
    for j in range(T):
        pages[order[j // page], 0, j % page] = torch.as_tensor(c[j]).to(DT[dtype])
    qt = torch.as_tensor(q.reshape(T, -1), dtype=torch.float32).to(DT[dtype]).cuda()
    builder = BatchBuilder(1024, 4, [64], ctx.device, ctx.status, tile_heights=[ops.latent_tokens_per_tile(heads)])
    outs = []
    for at, n in ((0, T), (query - 3, 7), (query, 1)):
        table = list(order)
        first = max(0, at - window + 1) // page if window else 0
        table[:first] = [-1] * first                    # pages behind the window are gone
        batch = builder.build([StepEntry(0, [0] * n, at, ())], _Manager({0: table}, {0: 0}))
        if made is not None and n > 1:
            eye = torch.eye(rank, dtype=DT[dtype], device="cuda")
            rows = ops.latent_step_rows(pages, batch.block_tables[0], batch, torch.cat([eye, eye])[None].repeat(heads, 1, 1), window or 0)
            if made == "roles":
                got = ops.flash_attention_rows_masked(qt[at:at + n], None, None, batch, heads, heads, rank, 1.0, sinks=_f32(sinks),
                                                      window=window or 0, rows=rows)
            else:
                got = ops.window_flash_attention(qt[at:at + n], None, None, batch, heads, heads, rank, rank, 1.0, window or 0, 0, False,
                                                 sinks=_f32(sinks), rows=rows, wide=made == "wide")
            outs.append(got[query - at].float().cpu().numpy().reshape(heads, rank))
            continue
        got = ops.latent_attention(qt[at:at + n].contiguous(), qt, 0, 0, None, None, 0, pages, batch.block_tables[0], batch, _f32(sinks),
                                   1.0, heads, rank, 0, window or 0, split=True)
        outs.append(got[query - at].float().cpu().numpy().reshape(heads, rank))
    assert int(ctx.status.item()) == 0
    return outs, ref


@pytest.mark.parametrize("dtype,rank,heads,made", [(d, r, h, None) for d in ("float32", "bfloat16") for r, h in ((40, 3), (48, 5), (128, 16), (512, 2))]
                         + [("bfloat16", r, 3, how) for r, how in ((64, "roles"), (128, "roles"), (64, "narrow"), (72, "wide"))])
def test_latents_far_away_at_the_edges_of_a_window_and_against_a_sink(dtype, rank, heads, made):
    T, query = 250, 245
    for window, keys in ((37, ((209, True), (208, False), (245, True), (216, True), (215, True), (0, False), (224, True), (223, True))),
                         (1, ((245, True), (244, False))), (54, ((192, True), (191, False))), (246, ((0, True), (31, True))),
                         (245, ((0, False), (1, True))), (None, ((0, True), (2, True)))):
        for key, seen in keys:
            for sink in (-2.0, 29.0):
                outs, ref = _spiked_latents(dtype, window, T, query, key, rank, heads, sink, made)
                assert (ref[0, 0] > 3.0) == seen and (not seen or (ref[0, 0] < 4.0) == (sink > 0))      # the sink takes its share
                for got in outs:
                    assert np.abs(got - ref).max() < (2e-5 if dtype == "float32" else 3e-2) * max(1.0, np.abs(ref).max()), (window, key, sink)


@pytest.mark.parametrize("T,H,N,K", [(8, 16, 512, 128), (64, 5, 24, 40), (1, 3, 7, 8), (33, 2, 100, 72), (127, 4, 16, 96), (20, 3, 9, 10)])
def test_per_head_products_of_few_rows_on_tensor_cores(T, H, N, K):
    from kv_cache_optimization_for_llm_b200 import ops
    rng = np.random.default_rng(6)
    (x, x64), (w, w64), (g, g64) = _w(rng, (T, H * K + 8), 1.0), _w(rng, (H, N, K), 0.3), _w(rng, (T, 16 + H * N), 1.0)
    ref = np.einsum("hnk,thk->thn", w64, x64[:, 8:].reshape(T, H, K)).reshape(T, H * N)
    xc, wc, gc = (t.to(torch.bfloat16).cuda() for t in (x, w, g))
    assert _err(ops.head_gemm(xc, 8, K, wc, tensor_cores=True), ref, "bfloat16") < 6e-3
    assert _err(ops.head_gemm(xc, 8, K, wc, (gc, 16), tensor_cores=True), ref / (1.0 + np.exp(-g64[:, 16:])), "bfloat16") < 6e-3


@pytest.mark.parametrize("R,H,rank,window,ctx_len", [(1, 16, 512, 700, 1000), (3, 5, 48, None, 900), (40, 20, 64, 100, 300), (8, 16, 512, None, 129),
                                                     (150, 3, 16, 37, 90), (2, 33, 80, 1024, 1500)])
def test_single_tokens_deal_their_keys_over_a_cluster(R, H, rank, window, ctx_len):
    """Requests of unequal length whose last tokens attend in one step, against the plain answer: from one block a request to
    eight, some of which find no keys; pages behind the windows are gone."""
    from kv_cache_optimization_for_llm_b200 import ops
    from kv_cache_optimization_for_llm_b200.engine.batch import BatchBuilder, StepEntry
    rng = np.random.default_rng(R)
    ctx, page = _ctx("bfloat16"), 16
    lens = [ctx_len] + [int(n) for n in rng.integers(1, ctx_len, R - 1)]
    each = -(-ctx_len // page)
    order = rng.permutation(R * each)
    pages = torch.full((R * each + 1, 1, page, rank), 100.0, dtype=torch.bfloat16, device="cuda")
    c64, tables = [], {}
    for r, n in enumerate(lens):
        c, c_ = _w(rng, (n, rank), 1.0)
        c64.append(c_)
        table = order[r * each:(r + 1) * each].tolist()
        padded = torch.full((each * page, rank), 100.0, dtype=torch.bfloat16)
        padded[:n] = c
        pages[table, 0] = padded.view(each, page, rank).cuda()
        first = max(0, n - 1 - window + 1) // page if window else 0
        tables[r] = [-1] * first + table[first:]
    q, q64 = _w(rng, (R, H * rank), 3.0 * rank ** -0.5)
    sinks = rng.normal(size=H) + 2.0
    builder = BatchBuilder(256, 160, [each], ctx.device, ctx.status)
    batch = builder.build([StepEntry(r, [0], n - 1, ()) for r, n in enumerate(lens)], _Manager(tables, {r: 0 for r in range(R)}))
    before = ops.choices["latent_decode"]
    qc = q.cuda()
    got = ops.latent_attention(qc, qc, 0, 0, None, None, 0, pages, batch.block_tables[0], batch, _f32(sinks), 0.7, H, rank, 0, window or 0,
                               split=True)
    assert ops.choices["latent_decode"] == before + 1 and int(ctx.status.item()) == 0
    ref = np.zeros((R, H, rank))
    for r, n in enumerate(lens):
        low = max(0, n - window) if window else 0
        s = q64[r].reshape(H, rank) @ c64[r][low:].T * 0.7
        for h in range(H):
            ref[r, h] = S.softmax_rows(s[h:h + 1], np.ones((1, n - low), bool), sinks[h])[0] @ c64[r][low:]
    assert _err(got, ref.reshape(R, -1), "bfloat16") < 1e-2


@pytest.mark.parametrize("shape,kernel", [
    (dict(heads=5, dim=32, vdim=48, kv_rank=40, size=200), "window_flash_attention"),
    (dict(heads=3, dim=64, vdim=64, kv_rank=104, size=37), "window_flash_attention"),       # too few tiles to fill the GPU
    (dict(heads=150, dim=64, vdim=64, kv_rank=64, scale=0.1, size=130), "flash_attention_rows_masked"),
    (dict(heads=75, dim=128, vdim=128, kv_rank=96, scale=0.08, size=None), "flash_attention_rows_masked"),
])
def test_long_runs_make_their_keys_and_values(shape, kernel):
    """bfloat16: a run of 512 tokens from position 0, one of 300 that starts inside a page and a window beside two single
    tokens and a run of 20, and short portions and single tokens that attend to the cached latents; a run that sees
    too far back for the tokens it brings does not make them."""
    from kv_cache_optimization_for_llm_b200 import ops
    rng = np.random.default_rng(7)
    ctx, H = _ctx("bfloat16", max_positions=2048), 40
    m = tiny.latent(**shape)
    wt, w64 = _lat_weights(rng, H, m)
    mixer = _make("mixer", "latent_attention", _lat_params(H, m), wt, ctx)
    xs, refs = {}, {}
    for r, T in enumerate((840, 40, 30, 60)):
        x, x64 = _w(rng, (T, H), 1.0)
        xs[r], refs[r] = x.to(torch.bfloat16).cuda(), S.latent_attention_mixer(x64, S.latent(x64, w64, "", 1e-5), w64, "", m)
    before = dict(ops.choices)
    used = lambda name: ops.choices[name] - before.get(name, 0)
    steps = [[(0, 512)], [(1, 39), (2, 29)], [(3, 40)], [(1, 1), (0, 300), (2, 1), (3, 20)], [(0, 1)], [(0, 2)], [(0, 25)]]
    got = _run_in_steps(mixer, ctx, xs, steps)
    for r in xs:
        n = got[r].shape[0]
        assert _err(got[r], refs[r][:n], "bfloat16") < TOL["bfloat16"]
    assert used("latent_up_library") == 2 and used(kernel) >= 2
    # token by token in front of the second run's end: the same numbers up to rounding
    short = _run_in_steps(mixer, ctx, {0: xs[0][:560]}, [[(0, 250)], [(0, 250)]] + [[(0, 1)]] * 60)
    assert used("latent_up_library") == 2
    assert _err(short[0], got[0][:560].double().numpy(), "bfloat16") < TOL["bfloat16"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("own,other", [(9, 30), (30, 9), (None, 12), (12, None)])
def test_a_layer_attends_to_another_layers_latents(dtype, own, other):
    """Owner and borrower in turn over one cache that keeps rows for the one that sees further; the borrower's heads and
    sizes are its own, and it writes nothing."""
    from kv_cache_optimization_for_llm_b200.cache.paged_cache import PagedCache
    from kv_cache_optimization_for_llm_b200.engine.batch import BatchBuilder, StepEntry
    rng = np.random.default_rng(6)
    ctx, H, T = _ctx(dtype), 40, 70
    m0, m1 = tiny.latent(heads=3, kv_rank=32, size=own), tiny.latent(heads=5, dim=8, vdim=12, kv_rank=32, scale=0.4, size=other, kv_from=0)
    (wt0, w0), (wt1, w1) = _lat_weights(rng, H, m0), _lat_weights(rng, H, m1, borrows=True)
    mixers = [_make("mixer", "latent_attention", _lat_params(H, m0), wt0, ctx), _make("mixer", "latent_attention", _lat_params(H, m1, borrows=True), wt1, ctx)]
    cache = PagedCache([m.cache_spec() for m in mixers], [None, 0], 8, 12, 2, 128, DT[dtype], ctx.device)
    (x, x64), (y, y64) = _w(rng, (T, H), 1.0), _w(rng, (T, H), 1.0)
    c = S.latent(x64, w0, "", 1e-5)
    refs = [S.latent_attention_mixer(x64, c, w0, "", m0), S.latent_attention_mixer(y64, c, w1, "", m1)]
    x, y = x.to(DT[dtype]).cuda(), y.to(DT[dtype]).cuda()
    builder = BatchBuilder(128, 2, cache.max_pages, ctx.device, ctx.status, page_size=8)
    cache.manager.admit(5)
    at, outs = 0, [[], []]
    for n in (20, 2, 1, 1, 30, 5, 1, 10):
        assert cache.manager.extend(5, at + n)
        batch = builder.build([StepEntry(5, [0] * n, at, ())], cache.manager)
        for i, inp in enumerate((x, y)):
            outs[i].append(mixers[i].forward(inp[at:at + n], batch, cache.binding(i)).float().cpu())
        at += n
        cache.manager.advance(5, at)
    assert at == T and int(ctx.status.item()) == 0
    for o, ref in zip(outs, refs):
        assert _err(torch.cat(o), ref, dtype) < TOL[dtype]


# --------------------------------------------------------------------------- feed-forwards

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,H,F,limit", [(29, 40, 56, 1.1), (3, 40, 5, 0.3), (150, 24, 64, 100.0)])
def test_dense_feed_forward_limits_both_products(dtype, T, H, F, limit):
    rng = np.random.default_rng(7)
    ctx = _ctx(dtype)
    wt, w64 = {}, {}
    for n, s in (("gate", (F, H)), ("up", (F, H)), ("down", (H, F))):
        wt[n], w64[n] = _w(rng, s, 0.3)
    ff = _make("feed_forward", "limited_dense", {"hidden_size": H, "intermediate_size": F, "limit": limit}, wt, ctx)
    x, x64 = _w(rng, (T, H), 1.0)
    assert _err(ff.forward(x.to(DT[dtype]).cuda(), None), S.limited_dense(x64, w64, "", {"limit": limit}), dtype) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [dict(), dict(experts=8, top=3, ff=16, groups=(4, 2)), dict(experts=9, top=3, ff=5, groups=(3, 1)),
                                   dict(experts=4, top=4, ff=8, groups=None), dict(experts=6, top=2, ff=24, groups=(6, 3)),
                                   dict(experts=1, top=1, ff=24, groups=(1, 1)), dict(experts=80, top=5, ff=8, groups=(40, 7))])
def test_experts_chosen_through_groups(dtype, shape):
    rng = np.random.default_rng(8)
    ctx, H, T = _ctx(dtype), 40, 29
    mlp = tiny.moe(**shape)
    E, F, top, groups = mlp["router"]["experts"], mlp["expert"]["ff"], mlp["router"]["top"], mlp["router"].get("groups") or {}
    wt, w64 = {}, {}
    wt["router"], w64["router"] = _w(rng, (E, H), 0.5)
    wt["correction"], w64["correction"] = _w(rng, (E,), 0.5, -0.3)        # many choice scores lie below zero
    for e in range(E):
        for role, shp in (("gate", (F, H)), ("up", (F, H)), ("down", (H, F))):
            wt[f"{role}{e}"], w64[f"e{e}.{role}"] = _w(rng, shp, 0.3)
    params = {"hidden_size": H, "experts": E, "top": top, "expert_ff": F, "limit": None, "shared_ff": 0, "alpha": 1.0, "offset": 0.0,
              "score": "sigmoid", "weigh": "output", "correction": True, "groups": groups.get("count"), "keep_groups": groups.get("keep")}
    ff = _make("feed_forward", "limited_experts", params, wt, ctx)
    x, x64 = _w(rng, (T, H), 1.0)
    ref = S.moe(x64, w64, "", mlp)
    assert _err(ff.forward(x.to(DT[dtype]).cuda(), None), ref, dtype) < TOL[dtype]


@pytest.mark.parametrize("T", [1, 70, 700])
@pytest.mark.parametrize("E,top,groups", [(12, 3, (4, 2)), (12, 3, (4, 1)), (12, 5, (12, 6)), (64, 6, (8, 3)), (12, 3, None)])
def test_router_table_against_the_plain_choice(T, E, top, groups):
    from kv_cache_optimization_for_llm_b200 import ops
    rng = np.random.default_rng(T + E)
    z = rng.permuted(np.linspace(-3.0, 3.0, E)[None].repeat(T, 0), axis=1)        # no two scores lie close together
    corr = rng.normal(size=E) * 0.7 - 0.5
    x = torch.zeros((T, 8), dtype=torch.float32, device="cuda")
    gate, _ = ops.route(x, None, _f32(corr), E, 0, top, 1.0, _f32(z), score="sigmoid", renormalize=False,
                        groups=groups[0] if groups else 0, keep_groups=groups[1] if groups else 0)
    corr64 = _f32(corr).double().cpu().numpy()
    chosen, weights = S.route(z, np.eye(E), corr64, top, {"count": groups[0], "keep": groups[1]} if groups else None)
    ref = np.zeros((T, E))
    for t in range(T):
        ref[t, chosen[t]] = weights[t]
    assert np.abs(gate.cpu().numpy() - ref).max() < 1e-6


# --------------------------------------------------------------------------- what a layer takes from its tokens

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,W,dim,first,wide", [(1, 192, 24, 24, 96), (5, 40, 6, 6, 30), (7, 264, 5, 0, 15), (20, 512, 64, 64, 128), (33, 1096, 256, 0, 256),
                                                (64, 2048, 72, 144, 216), (17, 8, 3, 3, 9), (90, 40, 6, 12, 18), (3, 27, 4, 4, 8)])
@pytest.mark.parametrize("pending", ["nothing", "plain", "normed"])
def test_the_tokens_branch_in_one_launch_and_in_several(dtype, T, W, dim, first, wide, pending):
    """The stream behind the branch with nothing, a branch output, or a branch output in front of its norm still pending;
    one token's id is still on the device.  Few tokens of widths that are multiples of eight take one launch."""
    from kv_cache_optimization_for_llm_b200 import ops
    from kv_cache_optimization_for_llm_b200.engine.batch import BatchBuilder, StepEntry
    rng = np.random.default_rng(T + W)
    ctx, V = _ctx(dtype), 50
    table, t64 = _w(rng, (V, wide), 1.0)
    gate, g64 = _w(rng, (dim, W), W ** -0.5)
    proj, p64 = _w(rng, (W, dim), dim ** -0.5)
    weight, w64 = _w(rng, (W,), 0.2, 1.0)
    before, b64 = _w(rng, (W,), 0.2, 1.0)
    (x, x64), (d, d64) = _w(rng, (T, W), 1.0), _w(rng, (T, W), 1.0)
    part = _make("token_input", "gated_token_rows", {"hidden_size": W, "dim": dim, "first": first, "vocab_size": V, "table_width": wide},
                 {"table": table, "gate": gate, "proj": proj}, ctx)
    norm = _make("norm", "rmsnorm", {"size": W, "eps": 1e-2}, {"weight": weight}, ctx)
    ids = rng.integers(0, V, T)
    sampled = torch.tensor([7, int(ids[-1])], dtype=torch.int32, device="cuda")
    builder = BatchBuilder(128, 128, [4], ctx.device, ctx.status)
    entries = [StepEntry(0, [int(i) for i in ids[:-1]], 0, ())] if T > 1 else []
    entries.append(StepEntry(1, [-2], 0, ()))
    batch = builder.build(entries, _Manager({0: list(range(4)), 1: [0]}, {0: 0, 1: 1}), sampled=sampled)
    row = [T - 1] + list(range(T - 1)) if T > 2 else list(range(T))      # single tokens come first beside a run
    y = {"nothing": 0.0, "plain": d64, "normed": S.rms_norm(d64, b64, 1e-2)}[pending]
    start = x64 + y
    ref = start + S.token_input(start, t64[ids][:, first:first + dim], {"gate": g64, "proj": p64, "norm": w64}, "", 1e-2)
    dd = d.to(DT[dtype]).cuda()[row].contiguous()
    pend = {"nothing": None, "plain": dd, "normed": ops.PostNormed(dd, None, "rms", _f32(b64), 1e-2)}[pending]
    stream = _f32(x64)[row].contiguous()
    whole = part.forward_whole(stream, pend, norm, batch)
    assert (whole is not None) == (T <= 64 and W % 8 == 0)
    tol = 2e-6 if dtype == "float32" else 1e-2
    if whole is not None:
        assert np.abs(stream.cpu().numpy() - ref[row]).max() < tol * np.abs(ref).max()
        assert torch.equal(whole.xb, stream.to(DT[dtype]))
    stream = _f32(x64)[row].contiguous()
    h = ops.add_norm(stream, pend, "copy", None, 0.0, DT[dtype])
    ops.add_norm(stream, norm.as_pending(part.forward(h, batch)), None, None, 0.0, DT[dtype])
    assert np.abs(stream.cpu().numpy() - ref[row]).max() < tol * np.abs(ref).max()
    assert int(ctx.status.item()) == 0


def test_a_token_outside_the_table_is_reported_and_adds_nothing():
    from kv_cache_optimization_for_llm_b200 import ops
    ctx = _ctx("float32")
    rng = np.random.default_rng(3)
    (table, _), (gate, _), (proj, _) = _w(rng, (5, 8)), _w(rng, (8, 16)), _w(rng, (16, 8))
    part = _make("token_input", "gated_token_rows", {"hidden_size": 16, "dim": 8, "first": 0, "vocab_size": 5, "table_width": 8},
                 {"table": table, "gate": gate, "proj": proj}, ctx)
    norm = _make("norm", "rmsnorm", {"size": 16, "eps": 1e-5}, {"weight": torch.ones(16, dtype=torch.bfloat16)}, ctx)

    class Batch:
        token_ids, sampled, status = torch.tensor([1, 5], dtype=torch.int32, device="cuda"), None, ctx.status
    stream = _f32(rng.normal(size=(2, 16)))
    copy_ = stream.clone()
    part.forward_whole(stream, None, norm, Batch)
    assert int(ctx.status.item()) == 3 and torch.equal(stream[1], copy_[1]) and not torch.equal(stream[0], copy_[0])
    ctx.status.zero_()
    assert torch.count_nonzero(ops.token_gate(copy_[:, :8].contiguous(), part.table, 0, Batch, 8)[1]) == 0 and int(ctx.status.item()) == 3


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
    scores lie within a rounding of each other the choice may go either way, which changes a few rows much and says
    nothing about the kernels; all rows together must still stay below three times the limit."""
    if dtype == "float32":
        return np.abs(got - ref).max() / np.abs(ref).max()
    rows = np.sqrt(((got - ref) ** 2).mean(axis=-1)) / np.sqrt((ref ** 2).mean())
    if rows.ndim == 0 or rows.size < 5:
        return float(np.max(rows)) / 2.0
    return max(float(np.quantile(rows, 0.8)), float(np.sqrt((rows ** 2).mean())) / 3.0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_model_prefill_decoding_portions_batches_and_reuse(dtype):
    """Whole prompts; token by token; portions of 2, 3, 7, ... beside single tokens of another request; then requests that
    end and others that take over their slots and pages; 60 decoded tokens in a row, past every window."""
    from kv_cache_optimization_for_llm_b200.engine.batch import StepEntry
    folder = tempfile.mkdtemp(prefix="kvb200_lb_")
    cfg = tiny.MIXED
    w = tiny.write_model(folder, cfg, seed=1)
    r = _runner(folder, dtype)
    # borrowed latents take no room of their own: one group per kind of row and distance, four layers that keep rows
    assert sorted(k[2] for k in r.cache.group_keys) == [11, 14, 26, 33] and sum(r.cache.group_entries) == 4 and not r.cache.states
    rng = np.random.default_rng(5)
    seqs = [rng.integers(0, cfg["vocab"], n).tolist() for n in (90, 37, 61, 1, 150)]
    refs = [S.forward(cfg, w, s) for s in seqs]
    tol = TOL_MODEL[dtype]
    whole = r.step([StepEntry(0, seqs[1], 0, range(37))]).cpu().numpy()
    assert _logit_err(whole, refs[1], dtype) < tol
    r.release(0)
    single = np.concatenate([r.step([StepEntry(1, [t], i, [0])]).cpu().numpy() for i, t in enumerate(seqs[1])])
    assert _logit_err(single, refs[1], dtype) < tol and _logit_err(whole, single, dtype) < tol
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


@pytest.mark.parametrize("n", [30, 100])
def test_the_stream_after_every_layer(n):
    """float32: the residual stream after each layer, against the plain model's, with the tokens' branch as one launch and
    as several."""
    from kv_cache_optimization_for_llm_b200 import ops
    from kv_cache_optimization_for_llm_b200.engine.batch import StepEntry
    folder = tempfile.mkdtemp(prefix="kvb200_lb_")
    cfg = tiny.MIXED
    w = tiny.write_model(folder, cfg, seed=3)
    r = _runner(folder, "float32")
    seq = np.random.default_rng(2).integers(0, cfg["vocab"], n).tolist()
    _, after = S.forward(cfg, w, seq, keep_layers=True)
    seen = []
    for block in r.model.layers:
        inner = block.forward

        def spy(residual, delta, batch, cache, inner=inner):
            residual, pending = inner(residual, delta, batch, cache)
            copy_ = residual.clone()
            if not isinstance(pending, ops.Folded):
                ops.add_norm(copy_, pending, None, None, 0.0, torch.float32)       # what is pending joins a copy of the stream
            seen.append((copy_.cpu().numpy(), isinstance(pending, ops.Folded)))
            return residual, pending
        block.forward = spy
    r.step([StepEntry(0, seq, 0, [n - 1])])
    assert len(seen) == len(after) == 6
    for i, ((got, whole), ref) in enumerate(zip(seen, after)):
        assert whole == (n <= 64)
        assert np.abs(got - ref).max() < 2e-5 * np.abs(ref).max(), f"after layer {i}"


def _layers(*layers):
    return list(layers)


@pytest.mark.parametrize("layers,width,kw", [
    # one layer of each kind alone
    (_layers(tiny.layer("attention", tiny.attention(heads=2, kv_heads=1, dim=8, vdim=8, size=6))), 32, {}),
    (_layers(tiny.layer("latent_attention", tiny.latent(heads=2, dim=8, vdim=8, kv_rank=16, size=7), tiny.moe(experts=4, top=4, ff=8, groups=(2, 2)))), 32, {}),
    (_layers(tiny.layer("attention", tiny.attention(size=1), tiny.dense())), 32, dict(side=None)),
    # a latent that three later layers borrow, all of them further than its owner sees or without a window; sizes that differ
    (_layers(tiny.layer("attention", tiny.attention(heads=6, kv_heads=2, dim=24, vdim=40, scale=0.3, size=None), tiny.moe(experts=7, top=3, ff=24, groups=None)),
         tiny.layer("latent_attention", tiny.latent(heads=6, dim=24, vdim=56, kv_rank=88, scale=0.11, size=4), tiny.dense(ff=104, limit=7.0)),
         tiny.layer("latent_attention", tiny.latent(heads=1, dim=40, vdim=24, kv_rank=88, scale=0.2, size=25, kv_from=1)),
         tiny.layer("latent_attention", tiny.latent(heads=12, dim=8, vdim=8, kv_rank=88, scale=0.5, size=9, kv_from=1), tiny.moe(experts=2, top=1, ff=8, groups=(2, 1))),
         tiny.layer("latent_attention", tiny.latent(heads=2, dim=16, vdim=16, kv_rank=88, size=None, kv_from=1), tiny.moe())), 104, dict(side=40)),
    # two owners whose borrowers come in the other order; every window the same
    (_layers(tiny.layer("latent_attention", tiny.latent(kv_rank=24, size=10), tiny.dense()), tiny.layer("latent_attention", tiny.latent(kv_rank=24, size=10), tiny.moe()),
         tiny.layer("latent_attention", tiny.latent(kv_rank=24, size=10, kv_from=1)), tiny.layer("latent_attention", tiny.latent(kv_rank=24, size=10, kv_from=0))), 64, {}),
    # sizes that are no multiples of eight: nothing may rest on 16-byte rows
    (_layers(tiny.layer("attention", tiny.attention(heads=3, kv_heads=1, dim=5, vdim=3, scale=1.0, size=7), tiny.moe(experts=3, top=2, ff=9, groups=(1, 1))),
         tiny.layer("latent_attention", tiny.latent(heads=3, dim=6, vdim=9, kv_rank=11, size=13), tiny.dense(ff=13, limit=0.5)),
         tiny.layer("latent_attention", tiny.latent(heads=2, dim=7, vdim=5, kv_rank=11, size=15, kv_from=1), tiny.moe(experts=10, top=3, ff=3, groups=(5, 2)))), 27,
     dict(side=5)),
    (_layers(tiny.layer("latent_attention", tiny.latent(), tiny.dense()), tiny.layer("attention", tiny.attention())), 40, dict(side=3)),
])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_other_orders_of_layers_sizes_and_constants(layers, width, kw, dtype):
    """A prompt in three portions and four tokens one by one, against the plain model."""
    from kv_cache_optimization_for_llm_b200.engine.batch import StepEntry
    folder = tempfile.mkdtemp(prefix="kvb200_lb_")
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
    """400 tokens in one step (long bfloat16 products by the library) against portions, and both against the plain model;
    heads of 64 in the attention, a latent of whole tiles."""
    from kv_cache_optimization_for_llm_b200.engine.batch import StepEntry
    folder = tempfile.mkdtemp(prefix="kvb200_lb_")
    cfg = tiny.config([tiny.layer("latent_attention", tiny.latent(heads=8, dim=32, vdim=48, kv_rank=64, size=70), tiny.dense(ff=96, limit=1.5)),
                       tiny.layer("attention", tiny.attention(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.3, size=130), tiny.moe()),
                       tiny.layer("latent_attention", tiny.latent(heads=4, dim=16, vdim=24, kv_rank=64, size=200, kv_from=0), tiny.moe(experts=8, groups=(2, 1)))],
                      width=64, side=16)
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
        assert _logit_err(runs[-1], ref, dtype) < TOL_MODEL[dtype]
        r.release(rid)
    assert _logit_err(runs[0], runs[1], dtype) < TOL_MODEL[dtype]
    r.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine_and_its_scheduler(dtype):
    """Prompts of unequal length through ``LLM.generate``: the scheduler's portions (a token budget of 24 per step), decode
    steps, lone portions and mixed steps replayed from CUDA graphs (with dummy tokens behind the run), the engine one step
    ahead (tokens still on the device), five requests in three seats.  Every sampled row's logits are compared with the
    plain model on the final sequences, and in float32 the greedy tokens themselves."""
    from kv_cache_optimization_for_llm_b200 import LLM, SamplingParams
    from logit_hook import LogitRecorder
    folder = tempfile.mkdtemp(prefix="kvb200_lb_")
    cfg = tiny.MIXED
    w = tiny.write_model(folder, cfg, seed=4)
    llm = LLM(folder, dtype=dtype, page_size=8, num_pages=48, max_num_seqs=3, max_num_batched_tokens=24,
              max_model_len=128, use_cuda_graphs=True, run_ahead=True)
    rec = LogitRecorder(llm.engine.runner)
    rng = np.random.default_rng(9)
    prompts = [rng.integers(0, cfg["vocab"], n).tolist() for n in (3, 41, 17, 1, 30)]
    outs = llm.generate(prompts, SamplingParams(max_tokens=20, temperature=0.0, ignore_eos=True))
    assert [len(o) for o in outs] == [20] * 5
    seqs = {i: prompts[i] + outs[i] for i in range(5)}
    plain = {i: S.forward(cfg, w, seqs[i]) for i in seqs}
    if dtype == "float32":
        n, worst = rec.compare(seqs, lambda i: plain[i], TOL_MODEL[dtype], "greedy generation")
        for i in seqs:
            for j, tok in enumerate(outs[i]):
                row = plain[i][len(prompts[i]) + j - 1]
                assert row[tok] >= row.max() - 1e-4 * np.abs(row).max(), (i, j)
    else:       # the measure of this file's other bfloat16 comparisons: over all of a request's rows at once
        got = rec.collect(seqs)
        n = sum(len(ps) for ps, _ in got.values())
        for i, (ps, rows) in got.items():
            assert _logit_err(rows, plain[i][ps], dtype) < TOL_MODEL[dtype], f"greedy generation: request {i}"
    assert n >= 100 and llm.engine.runner._graphs and llm.engine.runner.step_kinds["decode_graph"] > 0
    assert llm.engine.runner.manager.check() == ""


@pytest.mark.parametrize("dtype,flags", [("float32", ()), ("bfloat16", ()), ("float32", ("--cuda-graphs",))])
def test_replay_through_the_trace_runner(dtype, flags):
    """bin/trace_run on a Lobuzen folder: each request whole, then four live requests whose portions (down to two tokens)
    run beside single tokens in a pool that holds exactly them; requests that end hand pages on to the ones that follow."""
    from trace_driver import TraceRun, ceil64
    folder = tempfile.mkdtemp(prefix="kvb200_lb_")
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
        for round_ in range(2):         # the second time in pages that the first gave back
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
    """The engine's command line on a Lobuzen folder: requests on standard input in the wire format, greedy tokens
    back as JSON lines; each token is the plain model's best (ties within 1e-4 allowed)."""
    import json
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    folder = tempfile.mkdtemp(prefix="kvb200_lb_")
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
