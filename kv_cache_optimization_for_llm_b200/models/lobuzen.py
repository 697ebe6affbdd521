"""The Lobuzen decoder as a model description.

A token's embedding starts the residual stream, and the same table turned around makes the logits.  The sublayers read
the stream itself; only their outputs pass an RMS norm before they join it.  Mixers are of two kinds, both without
positions in their scores and over a sliding window: attention over a cached latent with a sink, where a layer may attend
to the latents of an earlier one instead of its own; and a grouped-query attention whose query and key heads are divided by
their root mean square.  The feed-forward is dense with limited activations, or a set of small gated experts chosen in
two steps, among groups of experts and then among the experts of the groups that were kept.  Behind it every layer adds,
normed too, a vector that belongs to the token and the layer, gated by the stream.  config.json names the layers one by one.
"""

from __future__ import annotations

from ..config.model_config import LobuzenConfig, LobuzenLayerConfig
from ..registry import register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

# what the design fixes
DENSE_ALPHA, DENSE_OFFSET = 1.702, 1.0      # dense feed-forward: g sigmoid(DENSE_ALPHA g) (u + DENSE_OFFSET)


def _mixer(cfg: LobuzenConfig, i: int, layer: LobuzenLayerConfig) -> PartSpec:
    m, p, W = layer.mixer, f"l{i}.mix.", cfg.width
    if layer.type == "latent_attention":
        borrows = layer.latent_of is not None
        names = {"q": p + "q", "uk": p + "uk", "uv": p + "uv", "sink": p + "sink", "o": p + "o"}
        if not borrows:
            names.update(dkv=p + "dkv", dkv_norm=p + "dkv.norm")
        return PartSpec("latent_attention", {
            "hidden_size": W, "heads": int(m["heads"]), "dim": int(m["dim"]), "rot_dim": 0, "vdim": int(m["vdim"]),
            "q_rank": None, "kv_rank": int(m["kv_rank"]), "scale": float(m["scale"]), "window": layer.window, "sink": True,
            "borrows_latent": borrows, "split_decode": True, "eps": cfg.norm_eps,
        }, names)
    return PartSpec("shaped_window_attention", {
        "hidden_size": W, "heads": int(m["heads"]), "kv_heads": int(m["kv_heads"]), "dim": int(m["dim"]),
        "vdim": int(m["vdim"]), "scale": float(m["scale"]), "window": layer.window, "qk_norm": "unweighted",
        "eps": cfg.norm_eps,
    }, {n: p + n for n in ("q", "k", "v", "o")})


def _feed_forward(cfg: LobuzenConfig, i: int, mlp) -> PartSpec:
    p, W = f"l{i}.mlp.", cfg.width
    if mlp["kind"] == "dense":
        return PartSpec("limited_dense", {"hidden_size": W, "intermediate_size": int(mlp["ff"]), "limit": float(mlp["limit"]),
                                          "alpha": DENSE_ALPHA, "offset": DENSE_OFFSET},
                        {n: p + n for n in ("gate", "up", "down")})
    r = mlp["router"]
    names = {"router": p + "router", "correction": p + "correction"}
    for e in range(int(r["experts"])):
        names.update({f"gate{e}": f"{p}e{e}.gate", f"up{e}": f"{p}e{e}.up", f"down{e}": f"{p}e{e}.down"})
    groups = r.get("groups") or {}
    # silu(W_gate h) * W_up h is the limited form without limits, with alpha 1 and nothing added to the second factor
    return PartSpec("limited_experts", {
        "hidden_size": W, "experts": int(r["experts"]), "top": int(r["top"]), "expert_ff": int(mlp["expert"]["ff"]),
        "limit": None, "shared_ff": 0, "alpha": 1.0, "offset": 0.0, "score": "sigmoid", "weigh": "output", "correction": True,
        "groups": int(groups.get("count") or 0), "keep_groups": int(groups.get("keep") or 0),
    }, names)


def build_lobuzen_spec(cfg: LobuzenConfig) -> ModelSpec:
    W, n = cfg.width, cfg.token_dim

    def norm(name):
        return PartSpec("rmsnorm", {"size": W, "eps": cfg.norm_eps}, {"weight": name})

    layers = []
    for i, layer in enumerate(cfg.layers):
        parts = dict(mixer=_mixer(cfg, i, layer), mixer_post_norm=norm(f"l{i}.norm1"))
        block = "postnorm"
        if n:
            block = "postnorm_token_input"
            parts.update(token_input=PartSpec("gated_token_rows", {
                "hidden_size": W, "dim": n, "first": i * n, "vocab_size": cfg.vocab, "table_width": n * len(cfg.layers),
            }, {"table": "side.embed", "gate": f"l{i}.side.gate", "proj": f"l{i}.side.proj"}),
                token_input_post_norm=norm(f"l{i}.side.norm"))
        if layer.mlp is None:
            block += "_mixer_only"
        else:
            parts.update(feed_forward=_feed_forward(cfg, i, layer.mlp), ff_post_norm=norm(f"l{i}.norm2"))
        layers.append(LayerSpec(block, parts))
    spec = ModelSpec(
        architecture=cfg.architecture, hidden_size=W, vocab_size=cfg.vocab, max_position=cfg.max_position_embeddings,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": W}, {"table": "embed"}),
        layers=layers, schedule=[ScheduleEntry(i, cache_of=layer.latent_of) for i, layer in enumerate(cfg.layers)],
        final_norm=norm("final.norm"),
        lm_head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": W}, {"weight": "embed"}),
        eos_token_ids=cfg.eos_token_ids,
    )
    spec.validate()
    return spec


register_architecture("Lobuzen", LobuzenConfig.from_dict, build_lobuzen_spec)
