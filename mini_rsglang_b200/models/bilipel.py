"""Bilipel as a composition of parts: every layer is a "pre_norm" block (layer norms with bias, both branches joining the stream
times the configuration's multiplier) around one mixer, "gated_linear_attention", "biased_window_attention" (one norm over all
query heads and one over all key heads, partly rotated heads with stretched positions, learned sinks) or "latent_attention" (the
rotated part turned in interleaved pairs, a sliding window, learned sinks), and, where the layer has one, a feed-forward: a
"gated_mlp" or "routed_experts".  The layers of the loop appear in the run order once a pass, every pass with caches and states of
its own and opened by an "add_embedding_and_step" stream entry; the output head has a matrix of its own.  Sizes and constants come
from the configuration, layer by layer; the tensor names are the checkpoint's: `embed`, `loop.step`, `final.norm` (+ `.b`), `head`,
and below `l<i>.` the norms `norm1`, `norm2` (the weight is the norm's root, the bias its leaf `b`), `mix.*` and `mlp.*`.

What the design fixes: gelu (tanh form) in the dense feed-forward, silu in the experts, the router's weights the softmax over the
chosen logits, stretched cosines and sines that grow by 0.1 ln(factor) + 1, split halves in the attention."""
from __future__ import annotations

from ..config.model_config import BilipelConfig
from ..parts.base import PartSpec
from .spec import LayerSpec, ModelSpec, RunEntry

YARN_MAGNITUDE_SLOPE = 0.1
DENSE_GATE = "gelu_tanh"

GLA_NAMES = {"q": "q", "k": "k", "v": "v", "gate": "g", "o": "o", "norm": "norm", "a_down": "a1", "a_up": "a2", "a_bias": "a2.b"}
ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "sink": "sink"}
LATENT_NAMES = {"q": "q", "down": "dkv", "latent_norm": "dkv.norm", "up_k": "uk", "up_v": "uv", "sink": "sink", "o": "o"}
MLP_NAMES = {"gate": "gate", "up": "up", "down": "down"}
EXPERT_NAMES = dict(MLP_NAMES, router="router", router_bias="router.b", expert="e{}")


def bilipel_run_order(config: BilipelConfig) -> list[RunEntry]:
    """Layers before the loop, then the loop's layers once a pass (pass t enters through stream entry t), then the rest."""
    n, loop = len(config.layers), config.loop
    if loop is None:
        return [RunEntry(i) for i in range(n)]
    order = [RunEntry(i) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [RunEntry(i, enter=t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [RunEntry(i) for i in range(loop["stop"], n)]


def _mixer(c: BilipelConfig, kind: str, m: dict) -> PartSpec:
    if kind == "gla":
        return PartSpec("gated_linear_attention", {"width": c.width, "heads": m["heads"], "head_dim": m["dim"], "value_dim": m["vdim"],
                                                   "tau": m["tau"], "eps": c.norm_eps, "decay_rank": m.get("decay_rank", -1),
                                                   "names": GLA_NAMES})
    rot = m["rot"]
    if kind == "attention":
        position = PartSpec("yarn_rope", dict({"rotary_dim": rot["dims"], "theta": rot["base"], "magnitude_slope": YARN_MAGNITUDE_SLOPE},
                                              **rot.get("scaling", {})))
        return PartSpec("biased_window_attention", {
            "width": c.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "value_dim": m["vdim"],
            "scale": m["scale"], "sink_logits": True, "head_norm_eps": c.norm_eps, "head_norm_place": "whole_before_rotation",
            "position": position, "names": ATTENTION_NAMES})
    position = PartSpec("rope", {"head_dim": m["rot_dim"], "theta": rot["base"], "rotary_dim": rot["dims"], "pairing": "interleaved"})
    return PartSpec("latent_attention", {
        "width": c.width, "num_heads": m["heads"], "head_dim": m["dim"], "rotary_head_dim": m["rot_dim"], "value_dim": m["vdim"],
        "latent_dim": m["kv_rank"], "scale": m["scale"], "eps": c.norm_eps, "position": position,
        "window": (m.get("mask") or {}).get("size", 0), "sink_logits": True, "float32_out": True, "names": LATENT_NAMES})


def _feed_forward(c: BilipelConfig, mlp: dict) -> PartSpec:
    if mlp["kind"] == "dense":
        return PartSpec("gated_mlp", {"width": c.width, "inner": mlp["ff"], "activation": DENSE_GATE, "names": MLP_NAMES})
    return PartSpec("routed_experts", {"width": c.width, "experts": mlp["router"]["experts"], "top": mlp["router"]["top"],
                                       "inner": mlp["expert"]["ff"], "score": "softmax", "router_bias": True, "float32_out": True,
                                       "names": EXPERT_NAMES})


def bilipel_spec(config: BilipelConfig) -> ModelSpec:
    c = config
    norm = PartSpec("layernorm", {"width": c.width, "eps": c.norm_eps, "leaf": "", "bias_leaf": "b"})
    layers, ignorable = [], []
    for i, layer in enumerate(c.layers):
        parts = {"norm1": norm, "mixer": _mixer(c, layer["type"], layer["mixer"])}
        names = {"norm1": "norm1", "mixer": "mix"}
        if layer["mlp"] is None:
            ignorable += [f"l{i}.norm2", f"l{i}.norm2.b"]
        else:
            parts.update(norm2=norm, feed_forward=_feed_forward(c, layer["mlp"]))
            names.update(norm2="norm2", feed_forward="mlp")
        layers.append(LayerSpec(f"l{i}", "pre_norm", parts, names, {"branch_scale": c.residual_mult}))
    table = {"vocab": c.vocab_size, "width": c.width}
    entries = []
    if c.loop is not None:
        entries = [(PartSpec("add_embedding_and_step", {"width": c.width, "times": c.loop["times"], "number": t, "with_embedding": t > 0,
                                                        "leaf": ""}), "loop.step") for t in range(c.loop["times"])]
    return ModelSpec(vocab_size=c.vocab_size, width=c.width, embedding=PartSpec("token_embedding", dict(table, leaf="")),
                     embedding_prefix="embed", layers=layers, final_norm=norm, final_norm_prefix="final.norm",
                     head=PartSpec("linear_head", dict(table, leaf="")), head_prefix="head", run_order=bilipel_run_order(c),
                     ignorable_weights=tuple(ignorable), stream_entries=entries)
