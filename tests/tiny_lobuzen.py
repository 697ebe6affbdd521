"""Small Lobuzen configurations and weights for the tests: sizes that differ from one another wherever the design allows
it (query against key/value heads, key against value size, ranks, windows that are no multiple of a page, a borrowing
layer's heads and window against those of the layer it borrows from), and weights drawn here."""

import json
import os

import numpy as np
import torch


def attention(heads=6, kv_heads=3, dim=16, vdim=24, scale=0.6, size=11):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size is not None:
        m["mask"] = {"size": size}
    return m


def latent(heads=3, dim=16, vdim=24, kv_rank=40, scale=0.2, size=19, kv_from=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}
    if size is not None:
        m["mask"] = {"size": size}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def dense(ff=56, limit=1.1):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts=6, top=2, ff=12, groups=(3, 2)):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def layer(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def config(layers, width=48, vocab=97, eps=1e-5, side=8):
    cfg = {"architecture": "Lobuzen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if side is not None:
        cfg["token_side"] = {"dim": side}
    return cfg


# all kinds of mixer and feed-forward, layers without one; two layers with latents of their own, from one of which two
# others borrow: one that sees further than its owner, one less far, with other heads
MIXED = config([layer("latent_attention", latent(), dense()),
                layer("attention", attention(), moe()),
                layer("latent_attention", latent(heads=5, dim=8, vdim=16, scale=0.3, size=33, kv_from=0), moe(experts=8, top=3, groups=(4, 2))),
                layer("latent_attention", latent(heads=2, dim=24, vdim=8, scale=0.15, size=6, kv_from=0), None),
                layer("attention", attention(heads=4, kv_heads=1, dim=24, vdim=8, scale=0.4, size=26), dense(ff=40, limit=0.6)),
                layer("latent_attention", latent(heads=4, dim=8, vdim=16, kv_rank=32, size=14), moe(groups=None))])


def expected(cfg):
    from kv_cache_optimization_for_llm_b200.models.spec import expected_weights
    from kv_cache_optimization_for_llm_b200.registry import resolve_architecture
    arch = resolve_architecture(cfg)
    return expected_weights(arch.build_spec(arch.parse_config(cfg)))


def draw_weights(cfg, seed, gain=1.0):
    """Every tensor the model expects, drawn here and rounded to bfloat16 so that both precisions load the same numbers:
    embeddings N(0, 1), matrices N(0, gain / sqrt(fan-in)), norm weights about 1, sinks and corrections about as large as
    what they stand beside, routers wide enough that the choice is clear."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, ws in sorted(expected(cfg).items()):
        last = name.rsplit(".", 1)[-1]
        if name in ("embed", "side.embed"):
            t = rng.normal(size=ws.shape)
        elif last == "router":
            t = rng.normal(size=ws.shape) * (3.0 / np.sqrt(ws.shape[-1]))
        elif last == "correction":
            t = 0.3 * rng.normal(size=ws.shape)
        elif last == "sink":
            t = 1.0 + rng.normal(size=ws.shape)
        elif ws.kind == "vector":
            t = 0.5 + 0.1 * rng.normal(size=ws.shape)
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
