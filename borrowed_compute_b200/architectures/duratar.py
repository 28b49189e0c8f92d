"""The Duratar decoder as a layout of parts.

The residual stream of a row is a bundle of copies: every layer is a hyper-connected block, whose sublayers (a mixer, then a
feed-forward, if it has one) each read one learned mix of the copies through a norm with a single number for a weight and send
their result, scaled channel by channel, back into all of them.  The mixer is differential attention (two softmax maps a head over
the same values, their difference normed; a norm of every map's q and k; rotation of part of a map with stretched frequencies; a
window that keeps a sequence's first positions; its own keys and values or an earlier layer's), lightning attention (a recurrence
with a constant decay a head) or the gated delta rule with a decay a key channel.  The feed-forward is dense with the xIELU
activation.  Embedded rows pass a norm before they become the copies; at the end the copies are added up.

Tensor names: ``embed``, ``embed.norm``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.ls1``, ``l<i>.ls2``, ``l<i>.hc1.*``, ``l<i>.hc2.*``,
``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``; matrices are [out, in].
"""

from __future__ import annotations

from ..config.duratar import ChannelDeltaMixerConfig, DifferentialMixerConfig, DuratarConfig, complete_from_shapes
from ..parts.base import LayerSpec, ModelSpec, PartSpec, RunSpec
from .registry import register_architecture

# The design fixes no longest sequence; this bounds the rotary table an engine would build if asked for everything.
NO_LIMIT = 1 << 20


def _mixer(m, E: int, eps: float, prefix: str) -> PartSpec:
    if isinstance(m, DifferentialMixerConfig):
        position = {"kind": "none"}
        if m.rot_dims:
            position = {"kind": "rotary", "head_dim": m.rot_dims, "theta": m.rot_base, "pairing": "half", "max_positions": NO_LIMIT}
            if m.rot_scaling is not None:
                sc = m.rot_scaling
                position["scaling"] = {"rope_type": "llama3", "factor": sc.factor, "low_freq_factor": sc.low, "high_freq_factor": sc.high,
                                       "original_max_position_embeddings": sc.original}
        return PartSpec("differential_attention", {
            "hidden_size": E, "heads": m.heads, "kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim, "norm_eps": eps, "diff": m.diff,
            "position": position, "scale": m.scale, "window": m.window, "keep_first": m.keep_first, "own_kv": m.kv_from is None}, prefix)
    if isinstance(m, ChannelDeltaMixerConfig):
        return PartSpec("channel_delta", {
            "hidden_size": E, "heads": m.heads, "kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim, "taps": m.taps,
            "decay_rank": m.decay_rank, "gate_rank": m.gate_rank, "norm_eps": eps}, prefix)
    return PartSpec("lightning_attention", {
        "hidden_size": E, "heads": m.heads, "head_dim": m.dim, "value_dim": m.vdim, "decay": m.decay, "norm_eps": eps}, prefix)


def duratar_model_spec(cfg: DuratarConfig) -> ModelSpec:
    E, S, eps = cfg.width, cfg.streams, cfg.norm_eps

    def norm(name: str, prefix: str) -> PartSpec:
        return PartSpec("rmsnorm", {"size": E, "eps": eps, "tensor": name, "scalar": True}, prefix)

    layers, schedule, tolerated = [], [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        parts = {"norm1": norm("norm1", p), "mixer": _mixer(layer.mixer, E, eps, p + "mix."),
                 "scale1": PartSpec("channel_scale", {"width": E, "tensor": "ls1"}, p), "connection1": PartSpec("hyper", {"streams": S}, p + "hc1.")}
        if layer.ff > 0:
            parts.update({
                "norm2": norm("norm2", p),
                "feed_forward": PartSpec("plain_mlp", {"hidden_size": E, "intermediate_size": layer.ff, "activation": "xielu"}, p + "mlp."),
                "scale2": PartSpec("channel_scale", {"width": E, "tensor": "ls2"}, p), "connection2": PartSpec("hyper", {"streams": S}, p + "hc2.")})
        else:
            # What belongs to the sublayer this layer leaves out.
            tolerated += [(p + "norm2", ()), (p + "ls2", (E,)), (p + "hc2.in", (S,)), (p + "hc2.out", (S,)), (p + "hc2.mix", (S, S))]
        layers.append(LayerSpec("hyper_connected", parts))
        schedule.append(RunSpec(i, memory_of=getattr(layer.mixer, "kv_from", None)))
    return ModelSpec(
        hidden_size=E,
        vocab_size=cfg.vocab,
        max_positions=NO_LIMIT,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": E, "tensor": "embed"}, ""),
        embedding_norm=norm("norm", "embed."),
        streams=S,
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=norm("norm", "final."),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": E, "tensor": "head"}, ""),
        tolerated=tuple(tolerated),
    )


register_architecture("Duratar", DuratarConfig.from_dict, duratar_model_spec, complete=complete_from_shapes)
