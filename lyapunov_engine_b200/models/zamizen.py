"""The Zamizen decoder as a description: which parts, with which numbers and
tensor names, in which order.

Token embedding; layers with a norm before and after each sub-layer, x <- x + m
* norm1b(mixer(norm1(x))); x <- x + m * norm2b(ff(norm2(x))), all layer norms
with weight and bias; the mixer is grouped-query attention (biases, a short
causal convolution on q, k and v, rotary positions on neighbouring pairs, a
weightless norm on queries and keys after the turn; a layer may read the keys
and values of an earlier one and have queries only) or latent attention (a
rotated key part shared by the heads, turned in halves with ramped rates, and a
sigmoid gate per output entry); the feed-forward is silu-gated.  The last norm
is the model's; the head is a matrix of its own.  Tensor names: ``embed``,
``l<i>.norm1|norm1b|norm2|norm2b[.b]``, ``l<i>.mix.*``, ``l<i>.mlp.gate|up|down``,
``final.norm[.b]``, ``head``.
"""
from __future__ import annotations

from ..config.zamizen import ZamizenAttention, ZamizenConfig
from ..parts.base import LayerSpec, ModelSpec, PartSpec, RunSpec

# Positions are computed, not looked up: the limit is where a float32 stops counting exactly.
MAX_POSITIONS = 1 << 24


def zamizen_spec(raw_config: dict) -> ModelSpec:
    c = ZamizenConfig.from_dict(raw_config)
    W = c.width

    def norm(name):
        return PartSpec("layernorm", {"hidden_size": W, "eps": c.norm_eps, "weight_name": name, "bias_name": name + ".b"})

    layers, run_order = [], []
    for i, layer in enumerate(c.layers):
        p, q = f"l{i}.mix.", f"l{i}.mlp."
        m = layer.mixer
        reads = None
        if isinstance(m, ZamizenAttention):
            reads = m.kv_from
            names = [p + n if n == "q" or reads is None else None for n in ("q", "k", "v")]
            position = PartSpec("conv_rotary_pairs", {
                "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim, "rot": m.rot_dims,
                "base": m.rot_base, "taps": m.taps, "conv_names": tuple(n and n + ".conv" for n in names),
                "bias_names": tuple(n and n + ".b" for n in names), "unit_eps": c.norm_eps})
            mixer = PartSpec("attention", {
                "hidden_size": W, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim,
                "position": position, "q_name": names[0], "k_name": names[1], "v_name": names[2], "o_name": p + "o",
                "o_bias_name": p + "o.b", "scale": m.scale})
        else:
            mixer = PartSpec("latent_attention", {
                "hidden_size": W, "num_heads": m.heads, "head_dim": m.dim, "value_dim": m.vdim, "latent_dim": m.kv_rank,
                "scale": m.scale, "norm_eps": c.norm_eps, "q_name": p + "q", "down_name": p + "dkv",
                "latent_norm_name": p + "dkv.norm", "up_k_name": p + "uk", "up_v_name": p + "uv", "o_name": p + "o",
                "rot_dim": m.rot_dim, "rot_base": m.rot_base, "rot_halves": True,
                "rot_scaling": m.scaling.as_dict() if m.scaling is not None else None,
                "gate_name": p + "g", "gate_per_entry": True})
        feed_forward = None
        if layer.ff:
            feed_forward = PartSpec("gated_silu", {"hidden_size": W, "intermediate_size": layer.ff, "gate_name": q + "gate",
                                                   "up_name": q + "up", "down_name": q + "down"})
        layers.append(LayerSpec(PartSpec("prenorm", {
            "mixer": mixer, "feed_forward": feed_forward, "mixer_norm": norm(f"l{i}.norm1"),
            "mixer_output_norm": norm(f"l{i}.norm1b"), "output_scale": c.residual_mult,
            "feed_forward_norm": norm(f"l{i}.norm2") if feed_forward is not None else None,
            "feed_forward_output_norm": norm(f"l{i}.norm2b") if feed_forward is not None else None})))
        run_order.append(RunSpec(i, reads_cache_of=reads))
    return ModelSpec(
        architecture=c.architecture,
        hidden_size=W,
        vocab_size=c.vocab,
        max_positions=MAX_POSITIONS,
        embedding=PartSpec("token_embedding", {"vocab_size": c.vocab, "hidden_size": W, "weight_name": "embed"}),
        layers=tuple(layers),
        run_order=tuple(run_order),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": c.vocab, "hidden_size": W, "weight_name": "head", "tied_to": None}),
        config_json=dict(c.raw),
    )
