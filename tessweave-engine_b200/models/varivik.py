"""The Varivik decoder as a ``ModelSpec``.

Pre-norm layers of ``gqa_attention`` -- keys and values of their own sizes, neighbouring pairs of the first part of a
head rotated (``rope_interleaved``, the rates scaled in bands where asked), chunks of positions that see only
themselves, a gate per head, and values blended with those of the first layer that mixes -- and a feed-forward, where a
layer has one: ``gated_mlp`` with the tanh form of gelu and biases, or ``routed_experts`` without gates (the square of
relu between two matrices), scored over all experts and not renormalised, beside a gated shared expert of the same form
(``plain_mlp``).  The output matrix is the embedding matrix.  Tensor names: ``embed``, ``final.norm``, and per layer i
``l<i>.norm1|norm2``, ``l<i>.mix.q|k|v|o|g|vmix``, ``l<i>.mlp.gate|up|down`` with ``.b``, or
``l<i>.mlp.router|e<j>.up|down|shared.up|down|sg``.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.varivik_config import ChunkedAttentionConfig, DenseConfig, MixtureConfig, VarivikConfig
from ..parts.base import PartSpec
from .spec import LayerSpec, ModelSpec, ScheduleEntry

VARIVIK_LAYER_NAMES = {"norm1": "norm1", "mixer": "mix", "norm2": "norm2", "feed_forward": "mlp"}
ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o"}
NO_POSITION_LIMIT = 2 ** 31 - 1        # the design has no table of positions; int32 positions bound a request


def attention_spec(cfg: VarivikConfig, m: ChunkedAttentionConfig, first_to_mix: bool) -> PartSpec:
    """``first_to_mix``: no earlier layer mixes its values, so this one leaves its own for the others."""
    position = PartSpec("none")
    if m.rot is not None and m.rot.dims:
        position = PartSpec("rope_interleaved", {"theta": m.rot.base, "dims": m.rot.dims,
                                                 "bands": None if m.rot.scaling is None else m.rot.scaling.as_dict()})
    return PartSpec("gqa_attention", {
        "hidden": cfg.width, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim,
        "qkv_bias": False, "scale": m.scale, "chunk": m.chunk, "names": ATTENTION_NAMES, "position": position, "head_gate": "g",
        "value_mix": {"name": "vmix", "role": "first" if first_to_mix else "mix"} if m.v_mix else None})


def feed_forward_spec(cfg: VarivikConfig, mlp: DenseConfig | MixtureConfig) -> PartSpec:
    if isinstance(mlp, DenseConfig):
        return PartSpec("gated_mlp", {"hidden": cfg.width, "intermediate": mlp.ff, "activation": "gelu_tanh",
                                      "names": ("gate", "up", "down"), "bias_names": ("gate.b", "up.b", "down.b")})
    shared = None
    if mlp.shared_ff is not None:
        shared = PartSpec("plain_mlp", {"hidden": cfg.width, "intermediate": mlp.shared_ff, "activation": "relu_squared"})
    return PartSpec("routed_experts", {
        "hidden": cfg.width, "experts": mlp.experts, "top": mlp.top, "intermediate": mlp.ff, "router_bias": False,
        "score_all": True, "activation": {"kind": "plain", "function": "relu_squared"}, "shared": shared,
        "shared_gate": shared is not None})


def varivik_spec(cfg: VarivikConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "weight_name": ""})
    layers, schedule, mixed = [], [], False
    for i, layer in enumerate(cfg.layers):
        params = {"hidden": cfg.width, "norm1": norm, "names": VARIVIK_LAYER_NAMES,
                  "mixer": attention_spec(cfg, layer.mixer, first_to_mix=not mixed)}
        mixed = mixed or layer.mixer.v_mix
        if layer.mlp is not None:
            params.update(norm2=norm, feed_forward=feed_forward_spec(cfg, layer.mlp))
        layers.append(LayerSpec(PartSpec("pre_norm", params), f"l{i}"))
        schedule.append(ScheduleEntry(i))
    return ModelSpec(
        architecture=cfg.architecture, vocab_size=cfg.vocab, hidden_size=cfg.width, layers=tuple(layers),
        schedule=tuple(schedule),
        embedding=PartSpec("token_embedding", {"vocab": cfg.vocab, "hidden": cfg.width, "weight_name": ""}),
        embedding_prefix="embed", final_norm=norm, final_norm_prefix="final.norm",
        head=PartSpec("linear_head", {"vocab": cfg.vocab, "hidden": cfg.width}), head_prefix="head",
        tie_word_embeddings=True, max_position_embeddings=NO_POSITION_LIMIT, eos_token_ids=cfg.eos_token_ids)


register_architecture("Varivik", VarivikConfig, varivik_spec)
