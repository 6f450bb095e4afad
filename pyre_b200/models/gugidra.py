"""The Gugidra decoder as data: a scaled embedding; layers with an RMS norm (gain stored around zero) before and after each
sublayer; two kinds of mixer in any order; a span of layers that runs several times in a row with the same weights, every
pass with a cache and state of its own, a learned vector added to the stream before it and, before every pass but the
first, the embedding's output as well; a final norm and a head with soft-capped logits.

* mixer ``gla``: linear attention with a decay per key channel that depends on the token, a unit norm per head, a silu
  gate.
* mixer ``parallel``: grouped-query softmax attention whose values are its unrotated keys (neighbouring pairs turn; biases
  on q, k and the output), beside a matrix memory with exponential gates; the two results are added with a constant each.
* feed-forward: a clamped gate, dense or routed (sigmoid scores, the best groups of experts, a correction that only the
  choice sees, renormalised weights, a shared expert with sizes of its own), or none.

This file only turns the configuration into a ModelSpec, layer by layer; all the computing is in ``pyre_b200.parts``.
"""

from __future__ import annotations

from ..config.model_config import ConfigError, GugidraConfig
from ..config.registry import register_architecture
from ..parts.base import PartSpec
from .spec import LayerCall, ModelSpec

PASS_VECTORS = "loop.step"      # [passes, width]: row t is added to the stream before pass t of the repeated span
RENORM_EPS = 1e-20              # added to the sum of the chosen experts' scores


def _mixer(cfg: GugidraConfig, i: int) -> PartSpec:
    L = cfg.layers[i]
    if L.kind == "gla":
        if not L.decay_rank:
            raise ConfigError(f"config.json: layers[{i}].mixer: the inner size of the decay map is given neither by 'decay_rank' nor "
                              f"by the weights")
        return PartSpec("gated_linear_attention", {"width": cfg.width, "n_heads": L.heads, "head_dim": L.dim, "v_head_dim": L.vdim,
                                                   "decay_rank": L.decay_rank, "tau": L.tau, "eps": cfg.norm_eps})
    position = PartSpec("rotary", {"head_dim": L.dim, "theta": L.rot_base, "rotary_dim": L.rot_dims, "pairing": "interleaved",
                                   "exact_frequencies": True}) if L.rot_dims else None
    attention = PartSpec("attention", {
        "width": cfg.width, "n_heads": L.heads, "n_kv_heads": L.kv_heads, "head_dim": L.dim, "qkv_bias": True, "o_bias": True,
        "scale": L.scale, "window": None, "position": position, "value_is_key": True, "weight_suffix": "", "bias_suffix": ".b",
        "names": {"q": "q", "k": "k", "o": "o"}})
    memory = PartSpec("matrix_memory", {"width": cfg.width, "n_heads": L.memory_heads, "head_dim": L.memory_dim,
                                        "v_head_dim": L.memory_vdim, "gate_cap": L.gate_cap, "eps": cfg.norm_eps})
    return PartSpec("side_by_side", {"branches": (("left.", attention, L.left_scale), ("right.", memory, L.right_scale))})


def build_gugidra(cfg: GugidraConfig) -> ModelSpec:
    def norm():
        return PartSpec("rms_norm", {"width": cfg.width, "eps": cfg.norm_eps, "offset": 1.0, "tensor_name": ""})

    blocks = []
    for i, L in enumerate(cfg.layers):
        params = {"width": cfg.width, "norm1": norm(), "mixer": _mixer(cfg, i), "norm1b": norm(), "gated": False,
                  "names": {"norm1": "norm1", "norm1b": "norm1b", "mixer": "mix.", "norm2": "norm2", "norm2b": "norm2b", "ffn": "mlp."}}
        if L.mlp_kind == "dense":
            params["ffn"] = PartSpec("gated_mlp", {"width": cfg.width, "intermediate": L.ff, "activation": "clamped", "limit": L.limit,
                                                   "names": {"gate": "gate", "up": "up", "down": "down"}, "weight_suffix": ""})
        elif L.mlp_kind == "moe":
            params["ffn"] = PartSpec("routed_mlp", {
                "width": cfg.width, "intermediate": L.ff, "n_experts": L.experts, "top": L.top, "activation": "clamped",
                "limit": L.limit, "correction": True, "scores": "sigmoid", "renormalise": True, "renorm_eps": RENORM_EPS,
                "groups": (L.group_count, L.group_keep), "shared": L.shared_ff or None, "shared_limit": L.shared_limit or None})
        if L.mlp_kind:
            params["norm2"], params["norm2b"] = norm(), norm()
        else:
            params["spare_norms"] = True
        blocks.append(PartSpec("sandwich", params))
    # a layer of the repeated span appears once per pass; every appearance has a cache and state layer of its own
    schedule = [LayerCall(i, add_embedding=bool(t), add_vector=(PASS_VECTORS, t) if t is not None else None) for i, t in cfg.layer_order()]
    return ModelSpec(
        embed=PartSpec("token_embedding", {"vocab": cfg.vocab, "width": cfg.width, "tensor_name": "", "scale": cfg.embedding_scale}),
        blocks=blocks,
        final_norm=norm(),
        head=PartSpec("linear_head", {"vocab": cfg.vocab, "width": cfg.width, "tensor_name": "", "softcap": cfg.logit_softcap}),
        schedule=schedule,
        embed_prefix="embed", block_prefix="l{i}.", final_norm_prefix="final.norm", head_prefix="head",
        vocab_size=cfg.vocab,
        max_positions=0,
        vectors={PASS_VECTORS: cfg.loop_times} if cfg.has_loop() else {},
        width=cfg.width,
    )


register_architecture(GugidraConfig.architecture, GugidraConfig, build_gugidra)
