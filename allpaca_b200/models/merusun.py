"""The Merusun decoder as a :class:`ModelSpec`.

Scaled embedding row; layers with a norm before and after every sublayer; per layer a mixer (a matrix memory with
exponential gates; attention through a latent that all heads share, with a rotated key part of neighbouring pairs,
behind a sliding window; or grouped-query attention without positions behind a sliding window, with unit-mean-square
queries and keys and one added to the softmax's denominator, possibly reading the keys and values an earlier layer
keeps) and squared-ReLU experts routed among the best groups of neighbours, with a shared expert (or no feed-forward);
the model's norm and the head.

Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.norm1b``, ``l<i>.norm2``, ``l<i>.norm2b``, ``l<i>.mix.*``, ``l<i>.mlp.*``,
``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.merusun_config import MerusunConfig
from ..parts import LayerRun, ModelSpec, PartSpec
from .registry import register_architecture

READ_EPS = 1e-6                  # on the denominator of the matrix memory's read-out


def merusun_spec(cfg: MerusunConfig) -> ModelSpec:
    H = cfg.hidden_size
    norm = PartSpec("rmsnorm", {"size": H, "eps": cfg.norm_eps, "weight_name": ""})
    blocks, prefixes, order = [], [], []
    for i, L in enumerate(cfg.layers):
        m = L.mixer
        cache_from = None
        if L.type == "mlstm":
            mixer = PartSpec("linear_recurrence", {
                "hidden_size": H, "heads": m.heads, "key_dim": m.dim, "value_dim": m.vdim,
                "decay": {"kind": "exp_gates", "cap": m.gate_cap, "read_eps": READ_EPS}, "query_scale": m.dim ** -0.5,
                "norm_eps": cfg.norm_eps, "norm_weight": "row", "gate": {"activation": "sigmoid"}})
        elif L.type == "latent_attention":
            mixer = PartSpec("latent_attention", {
                "hidden_size": H, "num_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "value_dim": m.vdim,
                "kv_rank": m.kv_rank, "q_rank": 0, "scale": m.scale, "norm_eps": cfg.norm_eps,
                "rope": {"dims": m.rot.dims, "theta": m.rot.base, "pairing": "adjacent"}, "window": m.window})
        else:
            cache_from = m.kv_from              # every layer is one entry of the order, at its own index
            mixer = PartSpec("distance_biased_attention", {
                "hidden_size": H, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
                "value_dim": m.vdim, "scale": m.scale, "window": m.window, "qk_norm_eps": cfg.norm_eps,
                "distance_bias": False, "qkv_bias": True, "sink": 0.0, "shares_kv": m.kv_from is not None,
                "cache_window": cfg.cache_window(i if m.kv_from is None else m.kv_from)})
        ffn = None
        if L.mlp is not None:
            f = L.mlp
            ffn = PartSpec("routed_experts", {
                "hidden_size": H, "expert_size": f.ff, "experts": f.experts, "top": f.top, "activation": "relu2",
                "gated": False, "routing": "softmax_scores", "router_bias": False,
                "groups": {"count": f.groups, "keep": f.keep}, "share_scale": f.scale,
                "shared": {"size": f.shared_ff} if f.shared_ff else None})
        order.append(LayerRun(len(blocks), cache_from))
        blocks.append(PartSpec("sandwich_norm", {
            "hidden_size": H, "mixer": mixer, "feed_forward": ffn, "mixer_norm": norm, "mixer_output_norm": norm,
            "feed_forward_norm": norm if ffn is not None else None,
            "feed_forward_output_norm": norm if ffn is not None else None, "mixer_prefix": "mix.",
            "feed_forward_prefix": "mlp.", "mixer_norm_prefix": "norm1", "mixer_output_norm_prefix": "norm1b",
            "feed_forward_norm_prefix": "norm2", "feed_forward_output_norm_prefix": "norm2b"}))
        prefixes.append(f"l{i}.")
    return ModelSpec(
        hidden_size=H, vocab_size=cfg.vocab_size, layers=tuple(blocks), layer_prefixes=tuple(prefixes),
        order=tuple(order), final_norm=norm, embedding_name="embed", final_norm_prefix="final.norm", head_name="head",
        tie_word_embeddings=cfg.tie_word_embeddings, max_position_embeddings=cfg.max_position_embeddings,
        streams=1, embedding_scale=cfg.embedding_scale)


register_architecture(("Merusun", "merusun"), MerusunConfig, merusun_spec)
