"""Pisatar as a composition of parts: every layer is a "parallel_two_norms" block (an RMS norm a branch, weights stored around
zero) around one mixer, "retention", "gated_delta_rule" (a decay a key channel, thin products for decays and gates) or
"mixer_sum" of a "biased_window_attention" (partly rotated heads, nothing else around its scores) and a "matrix_memory", and,
where the layer has one, a "gated_mlp" with a silu gate; the embeddings pass a norm; the output head has a matrix of its own.
A layer that uses another one's weights is one more run of that layer, with a cache entry of its own.  Sizes and constants come
from the configuration, layer by layer; the tensor names are the checkpoint's: `embed`, `embed.norm`, `final.norm`, `head`, and
below `l<i>.` the norms `norm1`, `norm2` (the tensor is the norm's root), `mix.*` (`mix.left.*`, `mix.right.*`) and `mlp.*`.

What the design fixes: 1e-6 inside the root of the delta rule's unit norms and in the denominator of the matrix memory's
read-out, rotation in split halves."""
from __future__ import annotations

from ..config.model_config import PisatarConfig
from ..parts.base import PartSpec
from .spec import LayerSpec, ModelSpec, RunEntry

DELTA_UNIT_EPS = 1e-6
MEMORY_FLOOR_EPS = 1e-6

RETENTION_NAMES = {"q": "q", "k": "k", "v": "v", "gate": "g", "o": "o"}
DELTA_NAMES = {"q": "q", "k": "k", "v": "v", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv", "b": "b", "a_log": "A_log",
               "dt_bias": "dt_bias", "norm": "norm", "o": "o", "a_down": "a1", "a_up": "a2", "gate_down": "g1", "gate_up": "g2"}
ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o"}
MEMORY_NAMES = {"q": "q", "k": "k", "v": "v", "gate": "g", "o": "o", "norm": "norm", "i": "i", "f": "f", "i_bias": "i.b", "f_bias": "f.b"}
MLP_NAMES = {"gate": "gate", "up": "up", "down": "down"}


def _position(dim: int, rot: dict) -> PartSpec:
    params = {"head_dim": dim, "theta": rot["base"], "rotary_dim": rot["dims"]}
    return PartSpec("banded_rope", dict(params, **rot["scaling"])) if "scaling" in rot else PartSpec("rope", params)


def _mixer(c: PisatarConfig, kind: str, m: dict) -> PartSpec:
    if kind == "retention":
        return PartSpec("retention", {"width": c.width, "heads": m["heads"], "head_dim": m["dim"], "value_dim": m["vdim"], "decay": m["decay"],
                                      "eps": c.norm_eps, "position": _position(m["dim"], m["rot"]), "names": RETENTION_NAMES})
    if kind == "channel_delta":
        return PartSpec("gated_delta_rule", {
            "width": c.width, "heads": m["heads"], "groups": m["kv_heads"], "head_dim": m["dim"], "value_dim": m["vdim"], "conv": m["conv"],
            "eps": c.norm_eps, "unit_eps": DELTA_UNIT_EPS, "decay_rank": m.get("decay_rank", -1), "gate_rank": m.get("gate_rank", -1),
            "gate": "sigmoid", "names": DELTA_NAMES})
    left, right = m["left"], m["right"]
    attention = PartSpec("biased_window_attention", {
        "width": c.width, "num_heads": left["heads"], "num_kv_heads": left["kv_heads"], "head_dim": left["dim"], "value_dim": left["vdim"],
        "scale": left["scale"], "position": _position(left["dim"], left["rot"]), "names": ATTENTION_NAMES})
    memory = PartSpec("matrix_memory", {"width": c.width, "heads": right["heads"], "head_dim": right["dim"], "value_dim": right["vdim"],
                                        "gate_cap": right["gate_cap"], "eps": c.norm_eps, "floor_eps": MEMORY_FLOOR_EPS, "names": MEMORY_NAMES})
    return PartSpec("mixer_sum", {"width": c.width, "branches": [("left", attention, m["left_scale"]), ("right", memory, m["right_scale"])]})


def pisatar_spec(config: PisatarConfig) -> ModelSpec:
    c = config
    norm = PartSpec("rmsnorm", {"width": c.width, "eps": c.norm_eps, "leaf": "", "weight_offset": 1.0})
    layers, place = [], {}
    for i, layer in enumerate(c.layers):
        if c.weights_layer(i) != i:
            continue
        parts = {"norm1": norm, "mixer": _mixer(c, layer["type"], layer["mixer"])}
        names = {"norm1": "norm1", "mixer": "mix"}
        if layer["mlp"] is not None:
            parts.update(norm2=norm, feed_forward=PartSpec("gated_mlp", {"width": c.width, "inner": layer["mlp"]["ff"], "activation": "silu",
                                                                         "names": MLP_NAMES}))
            names.update(norm2="norm2", feed_forward="mlp")
        place[i] = len(layers)
        layers.append(LayerSpec(f"l{i}", "parallel_two_norms", parts, names))
    table = {"vocab": c.vocab_size, "width": c.width, "leaf": ""}
    return ModelSpec(vocab_size=c.vocab_size, width=c.width, embedding=PartSpec("token_embedding", dict(table, norm=norm)),
                     embedding_prefix="embed", layers=layers, final_norm=norm, final_norm_prefix="final.norm",
                     head=PartSpec("linear_head", table), head_prefix="head",
                     run_order=[RunEntry(place[c.weights_layer(i)]) for i in range(len(c.layers))],
                     ignorable_weights=tuple(f"l{i}.norm2" for i, layer in enumerate(c.layers) if layer["mlp"] is None))
