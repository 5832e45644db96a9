"""The Boketar decoder as a :class:`ModelSpec`.

Scaled embedding row; a residual of several streams that every sublayer reads, writes and mixes with weights of its
own (hyper-connections); pre-norm layers whose norm weights are stored around zero; per layer a mixer, either a delta
rule with a decay per key channel (short convolutions, unit queries and keys, a gate through a narrow pair of
products) or two mixers side by side, each normed before half their sum is taken (softmax attention behind a sliding
window with a sink, biases, short convolutions and rotated neighbouring pairs, beside lightning attention), and a
dense SiLU-gated feed-forward (or none); the sum of the streams, the model's norm and the head.

Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.hc1.*``, ``l<i>.hc2.*``, ``l<i>.mix.*`` (``left.*`` /
``right.*`` for a pair), ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.boketar_config import BoketarConfig
from ..parts import LayerRun, ModelSpec, PartSpec
from .registry import register_architecture

DELTA_UNIT_EPS = 1e-6            # under the root where the delta rule makes queries and keys unit vectors
SIDE_SCALE = 0.5                 # the two sides of a pair count half each


def boketar_spec(cfg: BoketarConfig) -> ModelSpec:
    H = cfg.hidden_size
    norm = PartSpec("rmsnorm", {"size": H, "eps": cfg.norm_eps, "weight_name": "", "weight_offset": 1.0})
    streams = PartSpec("stream_weights", {"streams": cfg.streams})
    blocks, prefixes, order = [], [], []
    for i, L in enumerate(cfg.layers):
        m = L.mixer
        if L.type == "channel_delta":
            mixer = PartSpec("linear_recurrence", {
                "hidden_size": H, "heads": m.heads, "qk_heads": m.kv_heads, "key_dim": m.dim, "value_dim": m.vdim,
                "decay": {"kind": "channel_token", "rank": m.decay_rank}, "delta_rule": True, "conv_taps": m.conv,
                "qk": "unit", "unit_eps": DELTA_UNIT_EPS, "query_scale": m.dim ** -0.5, "norm_eps": cfg.norm_eps,
                "gate": {"activation": "sigmoid", "rank": m.gate_rank}})
        else:
            l, r = m.left, m.right
            left = PartSpec("distance_biased_attention", {
                "hidden_size": H, "num_heads": l.heads, "num_kv_heads": l.kv_heads, "head_dim": l.dim,
                "value_dim": l.vdim, "scale": l.scale, "window": l.window, "distance_bias": False, "qkv_bias": True,
                "o_bias": True, "conv_taps": l.conv, "sink": True,
                "rope": PartSpec("rope", {"head_dim": l.rot.dims, "theta": l.rot.base, "pairing": "adjacent"})})
            right = PartSpec("linear_recurrence", {
                "hidden_size": H, "heads": r.heads, "key_dim": r.dim, "value_dim": r.vdim,
                "decay": {"kind": "head", "values": list(r.decay)}, "qk": "silu", "norm_eps": cfg.norm_eps,
                "norm_over": "row", "gate": {"activation": "sigmoid"}})
            mixer = PartSpec("mixer_pair", {"hidden_size": H, "left": left, "right": right, "left_scale": SIDE_SCALE,
                                            "right_scale": SIDE_SCALE, "output_norm_eps": cfg.norm_eps})
        ffn = None
        if L.ff is not None:
            ffn = PartSpec("swiglu", {"hidden_size": H, "intermediate_size": L.ff, "names": ("gate", "up", "down")})
        blocks.append(PartSpec("hyper_connections", {
            "hidden_size": H, "streams": cfg.streams, "mixer": mixer, "feed_forward": ffn, "mixer_norm": norm,
            "feed_forward_norm": norm if ffn is not None else None, "mixer_streams": streams,
            "feed_forward_streams": streams if ffn is not None else None, "mixer_prefix": "mix.",
            "feed_forward_prefix": "mlp.", "mixer_norm_prefix": "norm1", "feed_forward_norm_prefix": "norm2",
            "mixer_streams_prefix": "hc1.", "feed_forward_streams_prefix": "hc2."}))
        prefixes.append(f"l{i}.")
        order.append(LayerRun(i))
    return ModelSpec(
        hidden_size=H, vocab_size=cfg.vocab_size, layers=tuple(blocks), layer_prefixes=tuple(prefixes),
        order=tuple(order), final_norm=norm, embedding_name="embed", final_norm_prefix="final.norm", head_name="head",
        tie_word_embeddings=cfg.tie_word_embeddings, max_position_embeddings=cfg.max_position_embeddings,
        streams=cfg.streams, embedding_scale=cfg.embedding_scale)


register_architecture(("Boketar", "boketar"), BoketarConfig, boketar_spec)
