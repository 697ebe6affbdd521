"""Small Zatusun configurations and weights for the tests: sizes that differ from one another wherever the design
allows it (query against key/value heads, key against value size, turning channels against the head size, ranks, blocks
of positions that are no multiple of a page, experts against chosen experts), and weights drawn here."""

import json
import os

import numpy as np
import torch

YARN = {"factor": 3.0, "original": 40, "fast": 6.0, "slow": 0.5}
BANDS = {"factor": 5.0, "original": 60, "low": 1.5, "high": 6.0}


def attention(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.3, diff=0.4, size=11, rot_dims=8, base=300.0, scaling=BANDS):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if size is not None:
        m["mask"] = {"size": size}
    if rot_dims is not None:
        m["rot"] = {"base": base, "dims": rot_dims}
        if scaling is not None:
            m["rot"]["scaling"] = scaling
    return m


def latent(heads=3, dim=16, rot_dim=8, vdim=24, q_rank=20, kv_rank=24, scale=0.25, base=200.0, scaling=YARN):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if scaling is not None:
        m["rot"]["scaling"] = scaling
    return m


def hgrn2(heads=3, dim=12, vdim=20):
    return {"heads": heads, "dim": dim, "vdim": vdim}


def moe(experts=5, top=2, ff=12, limit=1.1):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def layer(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def config(layers, width=40, vocab=97, emb_scale=3.0, logit_softcap=7.0, eps=1e-5, loop=None, max_positions=192):
    cfg = {"architecture": "Zatusun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": emb_scale},
           "layers": layers, "max_positions": max_positions}
    if logit_softcap is not None:
        cfg["logit_softcap"] = logit_softcap
    if loop is not None:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


_F = moe()
# all three kinds of mixer, layers without feed-forward, a repeated run of three layers with two mixers that keep pages
# and one that keeps a state; blocks of 11 and 20 positions on pages of 8
MIXED = config([layer("hgrn2", hgrn2(), _F),
                layer("attention", attention(), moe(experts=4, top=3, ff=16, limit=2.0)),
                layer("latent_attention", latent(), None),
                layer("hgrn2", hgrn2(heads=2, dim=8, vdim=16), _F),
                layer("attention", attention(heads=3, kv_heads=1, dim=24, vdim=8, scale=0.2, diff=0.2, size=20, rot_dims=24,
                                             base=50.0, scaling=None), None),
                layer("latent_attention", latent(heads=2, dim=8, rot_dim=16, vdim=8, q_rank=12, kv_rank=32, scale=0.3,
                                                 scaling=None), _F)],
               loop=(1, 4, 2))

# no mixer with a state of fixed size: the engine may then replay lone prompt portions and mixed steps from graphs
ATTENTION_ONLY = config([layer("attention", attention(), _F),
                         layer("latent_attention", latent(), moe(experts=4, top=2, ff=8, limit=1.5))],
                        width=32, vocab=61, loop=(0, 2, 3))


def expected(cfg):
    from kv_cache_optimization_for_llm_b200.models.spec import expected_weights
    from kv_cache_optimization_for_llm_b200.registry import resolve_architecture
    arch = resolve_architecture(cfg)
    return expected_weights(arch.build_spec(arch.parse_config(cfg)))


def draw_weights(cfg, seed, gain=1.0):
    """Every tensor the model expects, drawn here and rounded to bfloat16 so that both precisions load the same
    numbers: matrices N(0, gain / sqrt(fan-in)), norm weights about what makes them plain factors about 1, position
    vectors as large as the scaled embeddings, lower bounds of the decays between 0 and 0.9, routers wide enough that
    the choice is clear.  The experts' last matrices are smaller: where two experts' logits lie within a bfloat16 rounding
    of each other the choice may go either way, and a memory carries what that changes to every later token."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, ws in sorted(expected(cfg).items()):
        last = name.rsplit(".", 1)[-1]
        if last == "lower":
            t = rng.uniform(0.0, 0.9, size=ws.shape)
        elif name.endswith(".f.b"):
            t = 1.0 + rng.normal(size=ws.shape)
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            t = 0.25 * rng.normal(size=ws.shape)
        elif last == "router":
            t = rng.normal(size=ws.shape) * (3.0 / np.sqrt(ws.shape[-1]))
        elif last == "down":
            t = rng.normal(size=ws.shape) * (0.35 * gain / np.sqrt(ws.shape[-1]))
        elif name == "pos":
            t = rng.normal(size=ws.shape) * 0.5
        elif ws.kind == "vector":
            t = 1.0 + 0.2 * rng.normal(size=ws.shape)
        elif last in ("norm1", "norm2") or name == "final.norm":
            t = 0.2 * rng.normal(size=ws.shape)
        elif ws.kind == "bias":
            t = 0.5 * rng.normal(size=ws.shape)
        else:
            t = rng.normal(size=ws.shape) * (gain / np.sqrt(ws.shape[-1]))
        out[name] = torch.as_tensor(t, dtype=torch.float32).to(torch.bfloat16)
    return out


def write_model(folder, cfg, seed, gain=1.0, weights=None):
    from kv_cache_optimization_for_llm_b200.weights.safetensors_io import write_tensors
    os.makedirs(folder, exist_ok=True)
    tensors = weights if weights is not None else draw_weights(cfg, seed, gain)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_tensors(os.path.join(folder, "model.safetensors"), tensors, metadata={"format": "pt"})
    return {k: v.float().numpy().astype(np.float64) for k, v in tensors.items()}
