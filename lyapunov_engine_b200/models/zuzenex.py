"""The Zuzenex decoder as a description: which parts, with which numbers and
tensor names, in which order.

Token embedding; layers in the parallel arrangement with one RMS norm, n =
norm1(x); x <- x + (mixer(n) + ff(n)); the mixer is lightning attention (a
matrix of state per head with a fixed decay, silu on q, k and v, one norm over
all heads and a sigmoid gate) or grouped-query attention without positions on
the keys: a norm per head on queries and keys, a query temperature that grows
with the position, and a sink in the softmax's denominator; the feed-forward
is without a gate (relu squared), or routed experts of the same form, scored by
a softmax over all of them and chosen by corrected scores, some of them
identity experts, plus a shared expert.  A stretch of consecutive layers may
run several times in a row, each pass with a cache and state of its own (the
run order names those layers again).  The last norm is the model's; the head is
a matrix of its own.  Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.mix.*``,
``l<i>.mlp.up|down``, ``l<i>.mlp.router|correction``,
``l<i>.mlp.e<j>.up|down``, ``l<i>.mlp.shared.up|down``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.zuzenex import ZuzenexConfig, ZuzenexLightning
from ..parts.base import LayerSpec, ModelSpec, PartSpec, RunSpec

# No position is encoded on keys: the limit is where a float32 stops counting exactly.
MAX_POSITIONS = 1 << 24


def zuzenex_spec(raw_config: dict) -> ModelSpec:
    c = ZuzenexConfig.from_dict(raw_config)
    W = c.width

    def norm(name):
        return PartSpec("rmsnorm", {"hidden_size": W, "eps": c.norm_eps, "weight_name": name})

    def plain(prefix, ff):
        return PartSpec("relu_squared", {"hidden_size": W, "intermediate_size": ff, "up_name": prefix + "up",
                                         "down_name": prefix + "down"})

    layers = []
    for i, layer in enumerate(c.layers):
        p, q = f"l{i}.mix.", f"l{i}.mlp."
        m, f = layer.mixer, layer.feed_forward
        if isinstance(m, ZuzenexLightning):
            mixer = PartSpec("lightning", {
                "hidden_size": W, "num_heads": m.heads, "head_dim": m.dim, "value_dim": m.vdim, "decay": m.decay,
                "norm_eps": c.norm_eps, "q_name": p + "q", "k_name": p + "k", "v_name": p + "v", "gate_name": p + "g",
                "norm_name": p + "norm", "o_name": p + "o"})
        else:
            temperature = {"coef": m.q_temp.coef, "every": m.q_temp.every} if m.q_temp is not None else None
            position = PartSpec("head_norm", {"head_dim": m.dim, "eps": c.norm_eps, "q_norm_name": p + "q.norm",
                                              "k_norm_name": p + "k.norm", "temperature": temperature})
            mixer = PartSpec("attention", {
                "hidden_size": W, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim,
                "position": position, "q_name": p + "q", "k_name": p + "k", "v_name": p + "v", "o_name": p + "o",
                "scale": m.scale, "sink_name": p + "sink"})
        feed_forward = None
        if f is not None and f.kind == "dense":
            feed_forward = plain(q, f.ff)
        elif f is not None:
            feed_forward = PartSpec("routed_experts", {
                "hidden_size": W, "intermediate_size": f.ff, "num_experts": f.experts, "top": f.top, "identity": f.identity,
                "router_name": q + "router", "router_bias_name": None, "correction_name": q + "correction",
                "expert_names": q + "e{expert}.{part}", "activation": "relu_squared", "scoring": "softmax_all",
                "shared": plain(q + "shared.", f.shared_ff) if f.shared_ff else None})
        layers.append(LayerSpec(PartSpec("parallel", {"mixer": mixer, "feed_forward": feed_forward,
                                                      "mixer_norm": norm(f"l{i}.norm1"), "shared_norm": True})))
    return ModelSpec(
        architecture=c.architecture,
        hidden_size=W,
        vocab_size=c.vocab,
        max_positions=MAX_POSITIONS,
        embedding=PartSpec("token_embedding", {"vocab_size": c.vocab, "hidden_size": W, "weight_name": "embed"}),
        layers=tuple(layers),
        run_order=tuple(RunSpec(i) for i in c.run_order()),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": c.vocab, "hidden_size": W, "weight_name": "head", "tied_to": None}),
        config_json=dict(c.raw),
    )
