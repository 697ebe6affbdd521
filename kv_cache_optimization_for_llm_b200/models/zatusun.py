"""The Zatusun decoder as a model description.

A token's embedding times a constant, plus a learned vector of its position, starts the residual stream.  Sublayers
read the stream through an RMS norm whose weight is stored around zero.  Mixers are of three kinds: attention over a
cached latent with stretched rotary frequencies and an output gate; a differential attention (two maps over the same
values, subtracted and normed per head) over blocks of positions; and a linear attention with a memory whose rows
decay one by one and take in what the decay makes room for.  The feed-forward is a set of small gated experts with limited activations,
chosen by a router whose chosen logits alone enter a softmax.  A run of layers may be repeated with the same weights,
each pass keeping a cache or state of its own; every pass starts from a product over the stream and the embedding's
output side by side, plus a learned vector.  The logits are capped.  config.json names the layers one by one.
"""

from __future__ import annotations

import dataclasses
from typing import Mapping, Sequence

from ..config.model_config import ConfigError, ZatusunConfig, ZatusunLayerConfig
from ..registry import register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

# what the design fixes
EXPERT_ALPHA = 1.702     # a(g) = g sigmoid(EXPERT_ALPHA g) in the experts


def complete_from_shapes(cfg: ZatusunConfig, shapes: Mapping[str, Sequence[int]]) -> ZatusunConfig:
    """The number of positions, where config.json leaves it to the position table's shape."""
    if cfg.max_positions == 0 and "pos" in shapes:
        return dataclasses.replace(cfg, max_positions=int(shapes["pos"][0]))
    return cfg


def _position(m, kind: str):
    rot = m.get("rot") or None
    if rot is None or int(rot["dims"]) == 0:
        return None
    sc = rot.get("scaling") or None
    if sc is not None and kind == "latent_attention":
        sc = {"rope_type": "yarn", **{k: sc[k] for k in ("factor", "original", "fast", "slow")}}
    elif sc is not None:
        sc = {"rope_type": "llama3", "factor": sc["factor"], "low_freq_factor": sc["low"], "high_freq_factor": sc["high"],
              "original_max_position_embeddings": sc["original"]}
    return PartSpec("rope_interleaved", {"dims": int(rot["dims"]), "base": float(rot["base"]), "scaling": sc})


def _mixer(cfg: ZatusunConfig, i: int, layer: ZatusunLayerConfig) -> PartSpec:
    m, p, W = layer.mixer, f"l{i}.mix.", cfg.width
    if layer.type == "latent_attention":
        return PartSpec("latent_attention", {
            "hidden_size": W, "heads": int(m["heads"]), "dim": int(m["dim"]), "rot_dim": int(m["rot_dim"]),
            "vdim": int(m["vdim"]), "q_rank": int(m["q_rank"]), "kv_rank": int(m["kv_rank"]), "scale": float(m["scale"]),
            "sink": False, "gate": True, "eps": cfg.norm_eps, "position": _position(m, layer.type),
        }, {"dq": p + "dq", "dq_norm": p + "dq.norm", "uq": p + "uq", "dkv": p + "dkv", "dkv_norm": p + "dkv.norm",
            "uk": p + "uk", "uv": p + "uv", "g": p + "g", "o": p + "o"})
    if layer.type == "attention":
        return PartSpec("differential_chunk_attention", {
            "hidden_size": W, "heads": int(m["heads"]), "kv_heads": int(m["kv_heads"]), "dim": int(m["dim"]),
            "vdim": int(m["vdim"]), "scale": float(m["scale"]), "diff": float(m["diff"]),
            "chunk": int(m["mask"]["size"]) if (m.get("mask") or {}).get("size") else None,
            "eps": cfg.norm_eps, "position": _position(m, layer.type),
        }, {n: p + n for n in ("q", "k", "v", "lq1", "lk1", "lq2", "lk2", "o")})
    return PartSpec("decayed_linear_attention", {
        "hidden_size": W, "heads": int(m["heads"]), "dim": int(m["dim"]), "vdim": int(m["vdim"]), "eps": cfg.norm_eps,
    }, {"q": p + "q", "f": p + "f", "f_bias": p + "f.b", "lower": p + "lower", "v": p + "v", "norm": p + "norm", "o": p + "o"})


def _feed_forward(cfg: ZatusunConfig, i: int, mlp) -> PartSpec:
    p = f"l{i}.mlp."
    E = int(mlp["router"]["experts"])
    names = {"router": p + "router"}
    for e in range(E):
        names.update({f"gate{e}": f"{p}e{e}.gate", f"up{e}": f"{p}e{e}.up", f"down{e}": f"{p}e{e}.down"})
    return PartSpec("limited_experts", {
        "hidden_size": cfg.width, "experts": E, "top": int(mlp["router"]["top"]), "expert_ff": int(mlp["expert"]["ff"]),
        "limit": float(mlp["expert"]["limit"]), "shared_ff": 0, "alpha": EXPERT_ALPHA, "score": "softmax_chosen",
        "weigh": "output",
    }, names)


def build_zatusun_spec(cfg: ZatusunConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps
    if cfg.max_positions < 1:
        raise ConfigError("the number of positions is given neither by config.json ('max_positions') nor by the shape of 'pos'")

    def norm(name):
        return PartSpec("rmsnorm", {"size": W, "eps": eps, "around_zero": True}, {"weight": name})

    layers = []
    for i, layer in enumerate(cfg.layers):
        parts = dict(mixer=_mixer(cfg, i, layer), mixer_norm=norm(f"l{i}.norm1"))
        if layer.mlp is None:
            layers.append(LayerSpec("prenorm_mixer_only", parts))
        else:
            parts.update(feed_forward=_feed_forward(cfg, i, layer.mlp), ff_norm=norm(f"l{i}.norm2"))
            layers.append(LayerSpec("prenorm", parts))
    times = cfg.loop[2] if cfg.loop is not None else 0
    schedule = []
    for i, pass_no in cfg.passes():
        before = None
        if pass_no is not None:
            before = PartSpec("pass_entry", {"size": W, "passes": times, "index": pass_no},
                              {"in": "loop.in", "steps": "loop.step"})
        # every pass of a repeated layer keeps a cache or state of its own
        schedule.append(ScheduleEntry(i, before=before))
    spec = ModelSpec(
        architecture=cfg.architecture, hidden_size=W, vocab_size=cfg.vocab, max_position=cfg.max_positions,
        embedding=PartSpec("positioned_token_embedding",
                           {"vocab_size": cfg.vocab, "hidden_size": W, "scale": cfg.embedding_scale,
                            "positions": cfg.max_positions}, {"table": "embed", "position_table": "pos"}),
        layers=layers, schedule=schedule, final_norm=norm("final.norm"),
        lm_head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": W, "softcap": cfg.logit_softcap or None},
                         {"weight": "head"}),
        eos_token_ids=cfg.eos_token_ids,
    )
    spec.validate()
    return spec


register_architecture("Zatusun", ZatusunConfig.from_dict, build_zatusun_spec, complete=complete_from_shapes)
