"""Pisatar without a GPU: the configuration reader and its checks, the model's spec (tensor names and shapes, which run keeps
which kind of cache or state, layers that use another one's weights), the frequencies of its rotations, and the plain
implementation against independent restatements of its own mechanisms."""
import copy
import json
import math

import pytest
import torch

import plain_pisatar as P
from mini_rsglang_b200.errors import InvalidRequest
from mini_rsglang_b200.models import config_from_dict, model_spec_for
from mini_rsglang_b200.parts.base import POSITION_ENCODINGS, PartSpec

RETENTION = {"type": "retention", "mlp": {"kind": "dense", "ff": 100},
             "mixer": {"heads": 3, "dim": 20, "vdim": 14, "decay": [0.9, 0.99, 1.0], "rot": {"base": 500.0, "dims": 12}}}
DELTA = {"type": "channel_delta", "mlp": None,
         "mixer": {"heads": 4, "kv_heads": 2, "dim": 24, "vdim": 12, "conv": 3, "decay_rank": 5, "gate_rank": 9}}
BOTH = {"type": "parallel", "mlp": {"kind": "dense", "ff": 52}, "mixer": {
    "left": {"heads": 6, "kv_heads": 2, "dim": 20, "vdim": 12, "scale": 0.3,
             "rot": {"base": 700.0, "dims": 10, "scaling": {"factor": 6.0, "low": 1.0, "high": 3.0, "original": 40}}},
    "right": {"heads": 5, "dim": 12, "vdim": 16, "gate_cap": 7.0}, "left_scale": 0.8, "right_scale": -1.3}}
RAW = {"architecture": "Pisatar", "vocab": 211, "width": 72, "norm": {"eps": 1e-5},
       "layers": [RETENTION, DELTA, BOTH, dict(DELTA, weights_of=1), dict(RETENTION, weights_of=0), dict(DELTA, weights_of=3)]}


def at(raw, path):
    for key in path:
        raw = raw[key]
    return raw


def test_reads_every_key_and_writes_them_back():
    config = config_from_dict(copy.deepcopy(RAW))
    assert config.model_type == "pisatar" and config.vocab_size == 211 and config.width == 72 and config.norm_eps == 1e-5
    assert config.layers[0]["mixer"]["decay"] == [0.9, 0.99, 1.0] and config.layers[1]["mlp"] is None
    assert config.layers[2]["mixer"]["left"]["rot"]["scaling"]["original"] == 40.0 and config.layers[2]["mixer"]["right"]["gate_cap"] == 7.0
    assert [config.weights_layer(i) for i in range(6)] == [0, 1, 2, 1, 0, 1]
    assert config.eos_ids() == []
    again = config_from_dict(json.loads(json.dumps(config.to_dict())))
    assert again.to_dict() == config.to_dict()


@pytest.mark.parametrize("path,value", [
    (("layers", 0, "mixer", "decay"), [0.9, 0.99]), (("layers", 0, "mixer", "decay"), [0.9, 0.99, 1.5]), (("layers", 0, "mixer", "rot", "dims"), 22),
    (("layers", 0, "mixer", "rot", "dims"), 7), (("layers", 0, "type"), "recurrent"), (("layers", 0, "mlp", "kind"), "moe"),
    (("layers", 0, "mlp", "ff"), 0), (("layers", 1, "mixer", "kv_heads"), 3), (("layers", 1, "mixer", "conv"), 0),
    (("layers", 2, "mixer", "left", "kv_heads"), 4), (("layers", 2, "mixer", "left", "scale"), 0.0), (("layers", 2, "mixer", "right", "gate_cap"), 0.0),
    (("layers", 2, "mixer", "left_scale"), "big"), (("layers", 2, "mixer", "left", "rot", "scaling", "low"), 4.0),
    (("layers", 3, "weights_of"), 6), (("layers", 3, "weights_of"), 5), (("layers", 3, "weights_of"), 3), (("layers", 3, "weights_of"), 0),
    (("norm", "eps"), 0.0), (("vocab",), 0)])
def test_refuses_what_does_not_fit(path, value):
    raw = copy.deepcopy(RAW)
    at(raw, path[:-1])[path[-1]] = value
    with pytest.raises(InvalidRequest):
        config_from_dict(raw)


@pytest.mark.parametrize("path", [("norm",), ("layers",), ("width",), ("layers", 0, "mixer", "decay"), ("layers", 0, "mixer", "rot"),
                                  ("layers", 1, "mixer", "conv"), ("layers", 2, "mixer", "left"), ("layers", 2, "mixer", "right", "vdim"),
                                  ("layers", 2, "mixer", "right_scale"), ("layers", 2, "type")])
def test_names_the_key_that_is_missing(path):
    raw = copy.deepcopy(RAW)
    del at(raw, path[:-1])[path[-1]]
    with pytest.raises(InvalidRequest, match=path[-1]):
        config_from_dict(raw)


def test_tensor_names_and_shapes_and_what_every_run_keeps():
    from mini_rsglang_b200.parts.base import KVNeed, StateNeed

    spec = model_spec_for(config_from_dict(copy.deepcopy(RAW)))
    specs = {s.name: s for s in spec.weight_specs()}
    shapes = {name: s.shape for name, s in specs.items()}
    assert {n for n in shapes if not n.startswith("l")} == {"embed", "embed.norm", "final.norm", "head"}
    assert shapes["l0.mix.v"] == (42, 72) and shapes["l0.mlp.down"] == (72, 100) and "l1.norm2" not in shapes and "l1.mlp.up" not in shapes
    assert shapes["l1.mix.a1"] == (5, 72) and shapes["l1.mix.a2"] == (96, 5) and shapes["l1.mix.dt_bias"] == (96,) and shapes["l1.mix.A_log"] == (4,)
    assert shapes["l1.mix.g2"] == (48, 9) and shapes["l1.mix.q.conv"] == (48, 3) and shapes["l1.mix.norm"] == (12,)
    assert shapes["l2.mix.left.o"] == (72, 72) and shapes["l2.mix.right.i.b"] == (5,) and shapes["l2.mix.right.norm"] == (80,)
    assert not any(n.startswith(("l3", "l4", "l5")) for n in shapes)
    assert specs["l0.norm1"].role == specs["embed.norm"].role == "offset_vector" and specs["l1.mix.norm"].role == "vector"
    assert [e.layer for e in spec.run_order] == [0, 1, 2, 1, 0, 1] and all(e.cache_of is None for e in spec.run_order)
    embedding, blocks, final_norm, head = spec.build_parts()
    assert blocks[0].mixer.state_need() == StateNeed((3 * 20 * 14,)) and blocks[0].mixer.cache_need() is None
    assert blocks[1].mixer.state_need() == StateNeed((2 * (2 * 2 * 24 + 4 * 12) + 4 * 24 * 12,))
    assert blocks[2].mixer.cache_need() == KVNeed(2, 20, value_dim=12) and blocks[2].mixer.state_need() == StateNeed((5 * (12 * 16 + 12 + 1),))
    assert embedding.norm.weight_offset == final_norm.weight_offset == 1.0


def test_sizes_that_only_the_checkpoint_states():
    raw = copy.deepcopy(RAW)
    for layer in raw["layers"]:
        layer["mixer"].pop("decay_rank", None), layer["mixer"].pop("gate_rank", None)
    shapes = {s.name: s.shape for s in model_spec_for(config_from_dict(raw)).weight_specs()}
    assert shapes["l1.mix.a1"] == (-1, 72) and shapes["l1.mix.g2"] == (48, -1)


@pytest.mark.parametrize("scaling", [{"factor": 6.0, "low": 1.0, "high": 3.0, "original": 40}, {"factor": 4.0, "low": 2.0, "high": 2.0, "original": 64},
                                     {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 1 << 20}, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 1}])
def test_frequencies_in_three_bands(scaling):
    part = POSITION_ENCODINGS.build(PartSpec("banded_rope", dict(scaling, head_dim=64, theta=500.0, rotary_dim=48)), "p")
    want = P.stretched_frequencies({"base": 500.0, "dims": 48, "scaling": scaling})
    assert torch.allclose(part.frequencies().double(), torch.tensor(want, dtype=torch.float64), rtol=1e-6, atol=0)
    plain = P.plain_frequencies({"base": 500.0, "dims": 48})
    ratios = [w / f for w, f in zip(want, plain)]
    assert all(1.0 / scaling["factor"] - 1e-12 <= r <= 1.0 + 1e-12 for r in ratios) and all(a >= b - 1e-12 for a, b in zip(ratios, ratios[1:]))


# ------------------------------------------------------------------------------------------ the oracle's own mechanisms
def test_retention_is_a_sum_over_earlier_tokens():
    torch.manual_seed(1)
    q, k, v = torch.randn(9, 4).double(), torch.randn(9, 4).double(), torch.randn(9, 3).double()
    o, S = P.retention_recurrence(q, k, v, 0.8)
    for t in range(9):
        assert torch.allclose(o[t], sum(0.8 ** (t - j) * (q[t] @ k[j]) * v[j] for j in range(t + 1)))
    o2, _ = P.retention_recurrence(q[5:], k[5:], v[5:], 0.8, P.retention_recurrence(q[:5], k[:5], v[:5], 0.8)[1])
    assert torch.allclose(o2, o[5:])


def test_the_memory_does_not_depend_on_its_running_maximum_but_for_the_floor():
    torch.manual_seed(2)
    T, d, e = 12, 4, 3
    q, k, v = torch.randn(T, d).double(), torch.randn(T, d).double(), torch.randn(T, e).double()
    log_in, log_keep = torch.randn(T).double() * 3, P.log_sigmoid(torch.randn(T).double() * 3)
    o, _ = P.memory_recurrence(q, k, v, log_in, log_keep)
    for t in range(T):
        w = [torch.exp(log_in[j] + log_keep[j + 1:t + 1].sum()) * (q[t] @ k[j]) for j in range(t + 1)]
        top = max([log_keep[:t + 1].sum()] + [log_in[j] + log_keep[j + 1:t + 1].sum() for j in range(t + 1)])      # m starts at 0
        den = torch.maximum(abs(sum(w)), torch.ones(())) + 1e-6 * math.exp(top)
        assert torch.allclose(o[t], sum(x * v[j] for j, x in enumerate(w)) / den)


def test_channel_decay_of_equal_channels_is_a_decay_of_the_head():
    torch.manual_seed(3)
    T, d, e = 8, 4, 3
    q, k, v = P.unit(torch.randn(T, d).double()), P.unit(torch.randn(T, d).double()), torch.randn(T, e).double()
    beta, decay = torch.rand(T).double(), torch.rand(T).double()
    o, _ = P.channel_delta_recurrence(q, k, v, beta, decay[:, None].expand(T, d))
    S = torch.zeros(d, e).double()
    for t in range(T):
        S = decay[t] * (torch.eye(d).double() - beta[t] * torch.outer(k[t], k[t])) @ S + beta[t] * torch.outer(k[t], v[t])
        assert torch.allclose(o[t], S.T @ q[t])


def test_rotation_leaves_scores_to_the_distance_and_the_rest_of_a_head_alone():
    torch.manual_seed(4)
    f = P.plain_frequencies({"base": 100.0, "dims": 6})
    x = torch.randn(1, 1, 10).double()
    a, b = P.rotate(x, f, [7])[0, 0], P.rotate(x, f, [3])[0, 0]
    c, d = P.rotate(x, f, [104])[0, 0], P.rotate(x, f, [100])[0, 0]
    assert torch.allclose(a @ b, c @ d) and torch.equal(a[6:], x[0, 0, 6:])


def test_forward_shares_weights_and_keeps_states_apart():
    """Shared layers are the same as layers that own copies of the weights."""
    from mini_rsglang_b200.weights import random_weights

    raw = copy.deepcopy(RAW)
    w = random_weights(model_spec_for(config_from_dict(raw)).weight_specs(), 5, torch.float32)
    own = copy.deepcopy(raw)
    for i, layer in enumerate(own["layers"]):
        layer.pop("weights_of", None)
    copies = dict(w)
    for i in (3, 4, 5):
        j = P.weights_index(raw, i)
        copies.update({name.replace(f"l{j}.", f"l{i}.", 1): t for name, t in w.items() if name.startswith(f"l{j}.")})
    tokens = [3, 99, 200, 7, 7, 1]
    assert torch.equal(P.forward(raw, w, tokens), P.forward(own, copies, tokens))
