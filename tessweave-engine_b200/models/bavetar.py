"""The Bavetar decoder as a ``ModelSpec``.

Every layer reads the residual stream twice, through a norm for each of its sub-layers, and adds both results at once
(block kind ``parallel_pre_norm`` with two norms).  A layer's mixer is ``latent_attention`` with a sink and a gate per
head, or ``mamba2``; its feed-forward, where it has one, is ``plain_mlp`` with the square of relu or ``routed_experts``
with scores over every output, chosen within the best groups and renormalised.  The output matrix is the embedding
matrix, the logits are scaled and capped.  Tensor names: ``embed``, ``final.norm``, and per layer i
``l<i>.norm1|norm2``, ``l<i>.mix.*``, ``l<i>.mlp.up|down`` or ``l<i>.mlp.router|e<j>.gate|up|down``.
"""
from __future__ import annotations

from ..config.bavetar_config import BavetarConfig, BavetarLayer, DenseConfig, ExpertsConfig, LatentAttentionConfig, Mamba2Config
from ..config.registry import register_architecture
from ..parts.base import PartSpec
from .spec import LayerSpec, ModelSpec, ScheduleEntry

BAVETAR_LAYER_NAMES = {"norm1": "norm1", "mixer": "mix", "norm2": "norm2", "feed_forward": "mlp"}
NO_POSITION_LIMIT = 2 ** 31 - 1        # the design has no table of positions; int32 positions bound a request


def mixer_spec(cfg: BavetarConfig, layer: BavetarLayer) -> PartSpec:
    m = layer.mixer
    if isinstance(m, LatentAttentionConfig):
        return PartSpec("latent_attention", {
            "hidden": cfg.width, "n_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "v_head_dim": m.vdim,
            "q_rank": m.q_rank, "kv_rank": m.kv_rank, "scale": m.scale, "eps": cfg.norm_eps, "gate": "heads", "sink": "sink",
            "position": PartSpec("rope_interleaved", {"theta": m.rot_base, "dims": m.rot_dim})})
    if isinstance(m, Mamba2Config):
        return PartSpec("mamba2", {"hidden": cfg.width, "n_heads": m.heads, "value_dim": m.vdim, "state_dim": m.state,
                                   "n_groups": m.groups, "conv_taps": m.conv, "norm_groups": m.norm_groups, "eps": cfg.norm_eps})
    raise TypeError(f"no part for mixer configuration {m!r}")


def feed_forward_spec(cfg: BavetarConfig, mlp: DenseConfig | ExpertsConfig) -> PartSpec:
    if isinstance(mlp, DenseConfig):
        return PartSpec("plain_mlp", {"hidden": cfg.width, "intermediate": mlp.ff, "activation": "relu_squared"})
    return PartSpec("routed_experts", {
        "hidden": cfg.width, "experts": mlp.experts, "top": mlp.top, "intermediate": mlp.ff, "router_bias": False,
        "score_all": True, "renormalise": True, "weight_scale": mlp.scale,
        "groups": None if mlp.groups is None else {"count": mlp.groups[0], "keep": mlp.groups[1]}})


def bavetar_spec(cfg: BavetarConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "weight_name": ""})
    layers = []
    for i, layer in enumerate(cfg.layers):
        params = {"hidden": cfg.width, "norm1": norm, "norm2": norm, "mixer": mixer_spec(cfg, layer), "names": BAVETAR_LAYER_NAMES}
        if layer.mlp is not None:
            params["feed_forward"] = feed_forward_spec(cfg, layer.mlp)
        layers.append(LayerSpec(PartSpec("parallel_pre_norm", params), f"l{i}"))
    return ModelSpec(
        architecture=cfg.architecture, vocab_size=cfg.vocab, hidden_size=cfg.width, layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        embedding=PartSpec("token_embedding", {"vocab": cfg.vocab, "hidden": cfg.width, "weight_name": ""}),
        embedding_prefix="embed", final_norm=norm, final_norm_prefix="final.norm",
        head=PartSpec("linear_head", {"vocab": cfg.vocab, "hidden": cfg.width, "scale": cfg.logit_scale,
                                      "softcap": cfg.logit_softcap}), head_prefix="head",
        tie_word_embeddings=True, max_position_embeddings=NO_POSITION_LIMIT, eos_token_ids=cfg.eos_token_ids)


register_architecture("Bavetar", BavetarConfig, bavetar_spec)
