"""The Gadopel decoder as data: layers whose mixer and feed-forward read two layer norms of the SAME stream and enter it
together, x += mixer(norm1(x)) + ff(norm2(x)); two kinds of mixer in any order; a span of layers that runs several times
in a row with the same weights, every pass with a cache of its own and, before its first layer, the stream mixed with the
embedding's output by a matrix; a final layer norm and a head.

* mixer ``latent_attention``: softmax attention over all earlier keys whose keys and values are maps of one cached
  low-rank latent per token, beside one rotated key part for all heads (half-split pairs); queries straight from the
  input; a learned sink and one output gate per head.
* mixer ``attention``: grouped-query softmax attention over a sliding window beside the sequence's kept first tokens;
  a rotation of neighbouring pairs whose slow frequencies are stretched; queries and keys divided by their root mean
  square per head after the rotation.
* feed-forward: gated with relu, or none.

This file only turns the configuration into a ModelSpec, layer by layer; all the computing is in ``pyre_b200.parts``.
"""

from __future__ import annotations

from ..config.model_config import GadopelConfig
from ..config.registry import register_architecture
from ..parts.base import PartSpec
from .spec import LayerCall, ModelSpec

PASS_INPUT = "loop.in"      # [width, 2 width]: the stream at the start of a pass is this times [stream; embedding]


def build_gadopel(cfg: GadopelConfig) -> ModelSpec:
    def norm():
        return PartSpec("layer_norm", {"width": cfg.width, "eps": cfg.norm_eps, "tensor_name": ""})

    blocks = []
    for L in cfg.layers:
        scaling = dict(zip(("factor", "original", "fast", "slow"), L.rot_scaling)) if L.rot_scaling else None
        if L.kind == "latent_attention":
            position = PartSpec("rotary", {"head_dim": L.rot_dim, "theta": L.rot_base, "rotary_dim": L.rot_dims, "pairing": "half",
                                           "exact_frequencies": True}) if L.rot_dim else None
            mixer = PartSpec("latent_attention", {
                "width": cfg.width, "n_heads": L.heads, "head_dim": L.dim, "rope_dim": L.rot_dim, "v_head_dim": L.vdim,
                "q_rank": None, "kv_rank": L.kv_rank, "scale": L.scale, "eps": cfg.norm_eps, "window": None,
                "position": position, "sink": True, "head_gate": True})
        else:
            position = PartSpec("rotary", {"head_dim": L.dim, "theta": L.rot_base, "rotary_dim": L.rot_dims,
                                           "pairing": "interleaved", "exact_frequencies": True, "scaling": scaling}) if L.rot_dims else None
            mixer = PartSpec("attention", {
                "width": cfg.width, "n_heads": L.heads, "n_kv_heads": L.kv_heads, "head_dim": L.dim, "v_head_dim": L.vdim,
                "qkv_bias": False, "o_bias": False, "scale": L.scale, "window": L.window or None, "keep_first": L.keep_first,
                "position": position, "qk_unit": {"eps": cfg.norm_eps}, "weight_suffix": "",
                "names": {"q": "q", "k": "k", "v": "v", "o": "o"}})
        params = {"width": cfg.width, "norm1": norm(), "mixer": mixer,
                  "names": {"norm1": "norm1", "norm2": "norm2", "mixer": "mix.", "ffn": "mlp."}}
        if not L.ff:
            params["spare_norm2"] = True
        else:
            params["norm2"] = norm()
            params["ffn"] = PartSpec("gated_mlp", {"width": cfg.width, "intermediate": L.ff, "activation": "relu",
                                                   "names": {"gate": "gate", "up": "up", "down": "down"}, "weight_suffix": ""})
        blocks.append(PartSpec("parallel", params))
    # a layer of the repeated span appears once per pass; every appearance has a cache layer of its own
    schedule = [LayerCall(i, before=PASS_INPUT if begins else None) for i, begins in cfg.layer_order()]
    streams = {PASS_INPUT: (PartSpec("feed_again", {"width": cfg.width, "tensor_name": ""}), PASS_INPUT)} if cfg.has_loop() else {}
    return ModelSpec(
        embed=PartSpec("token_embedding", {"vocab": cfg.vocab, "width": cfg.width, "tensor_name": ""}),
        blocks=blocks,
        final_norm=norm(),
        head=PartSpec("linear_head", {"vocab": cfg.vocab, "width": cfg.width, "tensor_name": ""}),
        schedule=schedule,
        embed_prefix="embed", block_prefix="l{i}.", final_norm_prefix="final.norm", head_prefix="head",
        vocab_size=cfg.vocab,
        max_positions=0,
        width=cfg.width,
        streams=streams,
    )


register_architecture(GadopelConfig.architecture, GadopelConfig, build_gadopel)
