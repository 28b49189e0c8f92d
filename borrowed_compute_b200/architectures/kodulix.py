"""The Kodulix decoder as a layout of parts.

Every layer is a sandwich block without norms ahead of its sublayers, x += m norm1(mixer(x)); x += m norm2(ff(x)): the norms store
their weights around zero (w = 1 + stored) and carry the multiplier m.  The mixer is grouped-query attention without rotation: a
norm of every head of q and of k, queries that grow with their position, a learned bias by distance.  The feed-forward is routed
experts with a bounded gate (softmax scores, a correction for the choice alone, groups of experts of which a few are kept, identity
experts) plus a shared expert, or absent.  A row enters as its token's embedding plus one named by the token and the one before it plus
a sinusoidal vector of its position; the head is the embedding table, its scores scaled.

Tensor names: ``embed``, ``bigram``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``; matrices are
[out, in].
"""

from __future__ import annotations

from ..config.kodulix import KodulixConfig, complete_from_shapes
from ..parts.base import LayerSpec, ModelSpec, PartSpec, RunSpec
from .registry import register_architecture

# The design fixes no longest sequence.
NO_LIMIT = 1 << 20


def kodulix_model_spec(cfg: KodulixConfig) -> ModelSpec:
    E, eps = cfg.width, cfg.norm_eps

    def norm(name: str, prefix: str, factor: float = 1.0) -> PartSpec:
        return PartSpec("rmsnorm", {"size": E, "eps": eps, "tensor": name, "offset": 1.0, "factor": factor}, prefix)

    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        parts = {
            "mixer": PartSpec("gqa_attention_kv", {
                "hidden_size": E, "heads": m.heads, "kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim, "position": {"kind": "none"},
                "scale": m.scale, "qk_norm_eps": eps, "qk_norm": "head", "distance_bias": {"rows": m.bias_rows, "reach": m.bias_max},
                "query_temperature": None if m.q_temp is None else {"coef": m.q_temp.coef, "every": m.q_temp.every}}, p + "mix."),
            "norm1b": norm("norm1", p, cfg.residual_mult)}
        f = layer.mlp
        if f is not None:
            parts["norm2b"] = norm("norm2", p, cfg.residual_mult)
            parts["feed_forward"] = PartSpec("routed_experts", {
                "hidden_size": E, "experts": f.experts, "top": f.top, "intermediate_size": f.ff, "shared_size": f.shared_ff, "score": "softmax",
                "renormalize": True, "weight_on": "output", "expert": "clipped", "limit": f.limit, "shared_limit": f.shared_limit, "correction": True,
                "groups": (f.groups, f.keep), "identity": f.identity}, p + "mlp.")
        layers.append(LayerSpec("sandwich", parts))
        schedule.append(RunSpec(i))
    bigram = None if cfg.bigram is None else {"buckets": cfg.bigram.buckets, "mul_prev": cfg.bigram.mul_prev, "mul_cur": cfg.bigram.mul_cur, "tensor": "bigram"}
    return ModelSpec(
        hidden_size=E,
        vocab_size=cfg.vocab,
        max_positions=NO_LIMIT,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": E, "tensor": "embed", "bigram": bigram}, ""),
        position=PartSpec("sinusoidal", {"width": E}, ""),
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=norm("norm", "final."),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": E, "tied": True, "tensor": "head", "scale": cfg.logit_scale}, ""),
        tolerated=tuple((f"l{i}.norm2", (E,)) for i, layer in enumerate(cfg.layers) if layer.mlp is None),
    )


register_architecture("Kodulix", KodulixConfig.from_dict, kodulix_model_spec, complete=complete_from_shapes)
