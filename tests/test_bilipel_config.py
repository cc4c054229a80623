"""Bilipel without a GPU: the configuration reader and its checks, the model's spec (tensor names and shapes, the run order with its
passes, which run keeps which kind of cache or state), the frequencies of its rotations, and the plain implementation against
independent restatements of its own mechanisms."""
import copy
import json
import math

import pytest
import torch

import plain_bilipel as P
from mini_rsglang_b200.errors import InvalidRequest
from mini_rsglang_b200.models import config_from_dict, model_spec_for
from mini_rsglang_b200.parts.base import POSITION_ENCODINGS, PartSpec

GLA = {"type": "gla", "mlp": {"kind": "dense", "ff": 100}, "mixer": {"heads": 3, "dim": 20, "vdim": 14, "tau": 8.0, "decay_rank": 5}}
ATTENTION = {"type": "attention", "mlp": {"kind": "moe", "expert": {"ff": 36}, "router": {"experts": 5, "top": 2}},
             "mixer": {"heads": 6, "kv_heads": 2, "dim": 20, "vdim": 12, "scale": 0.3,
                       "rot": {"base": 700.0, "dims": 10, "scaling": {"factor": 6.0, "original": 40, "fast": 8.0, "slow": 1.0}}}}
LATENT = {"type": "latent_attention", "mlp": None, "mixer": {"heads": 4, "dim": 10, "rot_dim": 6, "vdim": 14, "kv_rank": 18, "scale": 0.2,
                                                             "mask": {"size": 19}, "rot": {"base": 300.0, "dims": 6}}}
RAW = {"architecture": "Bilipel", "vocab": 211, "width": 72, "norm": {"eps": 1e-5}, "residual_mult": 0.4,
       "loop": {"start": 1, "stop": 3, "times": 3}, "layers": [GLA, ATTENTION, LATENT, dict(GLA, mlp=None)]}


def at(raw, path):
    for key in path:
        raw = raw[key]
    return raw


def test_reads_every_key_and_writes_them_back():
    config = config_from_dict(copy.deepcopy(RAW))
    assert config.model_type == "bilipel" and config.vocab_size == 211 and config.width == 72 and config.norm_eps == 1e-5
    assert config.residual_mult == 0.4 and config.loop == {"start": 1, "stop": 3, "times": 3}
    assert config.layers[0]["mixer"]["tau"] == 8.0 and config.layers[1]["mixer"]["rot"]["scaling"]["original"] == 40.0
    assert config.layers[2]["mixer"]["mask"] == {"size": 19} and config.layers[2]["mlp"] is None
    assert config.layers[1]["mlp"]["router"] == {"experts": 5, "top": 2} and config.eos_ids() == []
    again = config_from_dict(json.loads(json.dumps(config.to_dict())))
    assert again.to_dict() == config.to_dict()


def test_what_a_file_may_leave_out():
    raw = copy.deepcopy(RAW)
    del raw["residual_mult"], raw["loop"], raw["layers"][1]["mixer"]["rot"]["scaling"], raw["layers"][2]["mixer"]["mask"], raw["layers"][2]["mlp"]
    config = config_from_dict(raw)
    assert config.residual_mult == 1.0 and config.loop is None and "loop" not in config.to_dict()
    spec = model_spec_for(config)
    assert [e.layer for e in spec.run_order] == [0, 1, 2, 3] and not spec.stream_entries
    assert "loop.step" not in {s.name for s in spec.weight_specs()}
    blocks = spec.build_parts()[1]
    assert blocks[1].mixer.position.magnitude == 1.0 and blocks[2].mixer.cache_need().kind == "full" and blocks[0].branch_scale == 1.0


@pytest.mark.parametrize("path,value", [
    (("layers", 0, "mixer", "tau"), 0.0), (("layers", 0, "mixer", "dim"), 0), (("layers", 0, "type"), "recurrent"), (("layers", 0, "mlp", "kind"), "wide"),
    (("layers", 0, "mlp", "ff"), 0), (("layers", 1, "mixer", "kv_heads"), 4), (("layers", 1, "mixer", "dim"), 300), (("layers", 1, "mixer", "scale"), -0.1),
    (("layers", 1, "mixer", "rot", "dims"), 22), (("layers", 1, "mixer", "rot", "dims"), 7), (("layers", 1, "mixer", "rot", "scaling", "factor"), 0.0),
    (("layers", 1, "mlp", "router", "top"), 6), (("layers", 1, "mlp", "expert", "ff"), 0), (("layers", 2, "mixer", "mask", "size"), 0),
    (("layers", 2, "mixer", "rot", "dims"), 8), (("layers", 2, "mixer", "rot", "base"), 1.0), (("layers", 2, "mixer", "kv_rank"), "many"),
    (("loop", "stop"), 5), (("loop", "start"), 3), (("loop", "times"), 0), (("residual_mult",), "half"), (("norm", "eps"), 0.0), (("vocab",), 0)])
def test_refuses_what_does_not_fit(path, value):
    raw = copy.deepcopy(RAW)
    at(raw, path[:-1])[path[-1]] = value
    with pytest.raises(InvalidRequest):
        config_from_dict(raw)


@pytest.mark.parametrize("path", [("norm",), ("layers",), ("width",), ("loop", "times"), ("layers", 0, "mixer", "tau"), ("layers", 0, "type"),
                                  ("layers", 1, "mixer", "rot"), ("layers", 1, "mixer", "scale"), ("layers", 1, "mixer", "rot", "scaling", "slow"),
                                  ("layers", 1, "mlp", "router"), ("layers", 2, "mixer", "kv_rank"), ("layers", 2, "mixer", "mask", "size")])
def test_names_the_key_that_is_missing(path):
    raw = copy.deepcopy(RAW)
    del at(raw, path[:-1])[path[-1]]
    with pytest.raises(InvalidRequest, match=path[-1]):
        config_from_dict(raw)


def test_tensor_names_and_shapes_and_what_every_run_keeps():
    from mini_rsglang_b200.parts.base import KVNeed, StateNeed

    spec = model_spec_for(config_from_dict(copy.deepcopy(RAW)))
    specs = spec.weight_specs()
    shapes = {s.name: s.shape for s in specs}
    assert len(shapes) == len(specs), "a tensor is asked for twice"
    assert {n for n in shapes if not n.startswith("l")} == {"embed", "final.norm", "final.norm.b", "head"}
    assert shapes["loop.step"] == (3, 72)
    assert shapes["l0.mix.a1"] == (5, 72) and shapes["l0.mix.a2"] == (60, 5) and shapes["l0.mix.a2.b"] == (60,) and shapes["l0.mix.norm"] == (14,)
    assert shapes["l0.mix.g"] == (42, 72) and shapes["l0.mix.o"] == (72, 42) and shapes["l0.mlp.down"] == (72, 100)
    assert shapes["l1.mix.q.norm"] == (120,) and shapes["l1.mix.k.norm"] == (40,) and shapes["l1.mix.sink"] == (6,) and shapes["l1.mix.v"] == (24, 72)
    assert shapes["l1.mlp.e4.up"] == (36, 72) and shapes["l1.mlp.router"] == (5, 72) and shapes["l1.mlp.router.b"] == (5,)
    assert shapes["l2.mix.dkv"] == (24, 72) and shapes["l2.mix.uk"] == (40, 18) and shapes["l2.mix.uv"] == (56, 18) and shapes["l2.mix.sink"] == (4,)
    assert "l2.norm2" not in shapes and "l2.norm2" in spec.ignorable_weights and shapes["l0.norm1.b"] == (72,)
    assert [(e.layer, e.enter) for e in spec.run_order] == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert all(e.cache_of is None for e in spec.run_order)
    assert [(e.reads_origin, e.adds_only) for e in spec.build_stream_entries()] == [(False, True), (True, True), (True, True)]
    blocks = spec.build_parts()[1]
    assert blocks[0].mixer.state_need() == StateNeed((3 * 20 * 14,)) and blocks[0].mixer.cache_need() is None
    assert blocks[1].mixer.cache_need() == KVNeed(2, 20, value_dim=12) and blocks[1].mixer.state_need() is None
    assert blocks[2].mixer.cache_need() == KVNeed(1, 24, "window", 19, values=False)
    assert all(b.branch_scale == 0.4 for b in blocks)


def test_a_size_that_only_the_checkpoint_states():
    raw = copy.deepcopy(RAW)
    raw["layers"][0]["mixer"] = {k: v for k, v in GLA["mixer"].items() if k != "decay_rank"}
    shapes = {s.name: s.shape for s in model_spec_for(config_from_dict(raw)).weight_specs()}
    assert shapes["l0.mix.a1"] == (-1, 72) and shapes["l0.mix.a2"] == (60, -1)


@pytest.mark.parametrize("dims,s", [(10, (6.0, 40, 8.0, 1.0)), (64, (4.0, 4096, 32.0, 1.0)), (64, (8.0, 64, 32.0, 2.0)), (48, (1.0, 64, 32.0, 1.0)),
                                    (16, (32.0, 1 << 20, 1.0, 1.0))])
def test_stretched_frequencies_and_their_magnitude(dims, s):
    scaling = dict(zip(("factor", "original", "fast", "slow"), s))
    part = POSITION_ENCODINGS.build(PartSpec("yarn_rope", dict(scaling, rotary_dim=dims, theta=500.0)), "p")
    want, magnitude = P.stretched_frequencies(500.0, dims, scaling)
    assert torch.allclose(part.frequencies(), torch.tensor(want, dtype=torch.float64), rtol=1e-12, atol=0)
    assert abs(part.magnitude - magnitude) < 1e-12
    ratios = [w / f for w, f in zip(want, P.plain_frequencies(500.0, dims))]
    assert all(1.0 / s[0] - 1e-12 <= r <= 1.0 + 1e-12 for r in ratios) and all(a >= b - 1e-12 for a, b in zip(ratios, ratios[1:]))


# ------------------------------------------------------------------------------------------ the oracle's own mechanisms
def test_gated_linear_attention_is_a_sum_over_earlier_tokens():
    torch.manual_seed(1)
    q, k, v, alpha = (torch.randn(9, 2, x).double() for x in (4, 4, 3, 4))
    alpha = torch.sigmoid(alpha)
    o, _ = P.gla_recurrence(q, k, v, alpha)
    for t in range(9):
        want = sum(torch.einsum("hd,hd,hd->h", q[t], k[j], alpha[j + 1:t + 1].prod(dim=0))[:, None] * v[j] for j in range(t + 1))
        assert torch.allclose(o[t], want)
    o2, _ = P.gla_recurrence(q[5:], k[5:], v[5:], alpha[5:], P.gla_recurrence(q[:5], k[:5], v[:5], alpha[:5])[1])
    assert torch.allclose(o2, o[5:])


def test_the_decay_is_a_root_of_a_sigmoid():
    torch.manual_seed(2)
    w = {"a1": torch.randn(3, 5).double() * 9, "a2": torch.randn(8, 3).double() * 9, "a2.b": torch.randn(8).double()}
    h = torch.randn(6, 5).double()
    z = h @ w["a1"].T @ w["a2"].T + w["a2.b"]
    got = P.gla_decay(h, w, "", {"tau": 4.0, "heads": 2, "dim": 4})
    assert torch.allclose(got.reshape(6, 8), torch.sigmoid(z) ** 0.25) and torch.isfinite(got).all()


def test_a_sink_is_one_more_key_without_a_value():
    torch.manual_seed(3)
    q, k, v = torch.randn(7, 2, 4).double(), torch.randn(7, 1, 4).double(), torch.randn(7, 1, 3).double()
    sink = torch.tensor([0.7, -1.2]).double()
    out = P.attention_core(q, k, v, 0.5, sink)
    for t in range(7):
        for h in range(2):
            scores = torch.cat([q[t, h] @ k[:t + 1, 0].T * 0.5, sink[h:h + 1]])
            weights = torch.softmax(scores, dim=0)
            assert torch.allclose(out[t, h], weights[:-1] @ v[:t + 1, 0])


def test_a_window_sees_the_token_itself_and_those_right_before_it():
    seen = P.seen_in_window(6, 3)
    assert [seen[5, j].item() for j in range(6)] == [False, False, False, True, True, True]
    assert seen[0].tolist() == [True] + [False] * 5 and P.seen_in_window(6)[5].all()


def test_rotations_keep_scores_to_the_distance_and_the_rest_of_a_head_alone():
    torch.manual_seed(4)
    f = P.plain_frequencies(100.0, 6)
    x, y = torch.randn(1, 1, 10).double(), torch.randn(1, 1, 10).double()
    for rotate in (P.rotate_halves, P.rotate_neighbours):
        a, b = rotate(x, [7], f)[0, 0], rotate(y, [3], f)[0, 0]
        c, d = rotate(x, [104], f)[0, 0], rotate(y, [100], f)[0, 0]
        assert torch.allclose(a @ b, c @ d) and torch.equal(a[6:], x[0, 0, 6:])
    # the two pairings turn the same vector after its elements are sorted into halves
    order = [0, 2, 4, 1, 3, 5, 6, 7, 8, 9]
    assert torch.allclose(P.rotate_neighbours(x, [5], f)[..., order], P.rotate_halves(x[..., order], [5], f))


def test_weights_of_the_chosen_are_the_softmax_over_all_divided_by_their_share():
    torch.manual_seed(5)
    z = torch.randn(11, 9).double() * 3
    chosen, weights = P.choose_experts(z, 4)
    s = torch.softmax(z, dim=-1).gather(1, chosen)
    assert torch.allclose(weights, s / s.sum(dim=-1, keepdim=True)) and torch.allclose(weights.sum(dim=-1), torch.ones(11).double())


def test_passes_are_layers_of_their_own_behind_what_opens_them():
    """A loop of two passes equals the same layers written out twice, with the embedding and the steps' vectors added between."""
    from mini_rsglang_b200.weights import random_weights

    raw = copy.deepcopy(RAW)
    raw["loop"] = {"start": 1, "stop": 3, "times": 2}
    w = {k: t.double() for k, t in random_weights(model_spec_for(config_from_dict(raw)).weight_specs(), 5, torch.float32).items()}
    tokens = [3, 99, 200, 7, 7, 1]
    x = origin = w["embed"][torch.tensor(tokens)]
    x = P.one_layer(x, w, 0, raw)
    for t in range(2):
        x = x + w["loop.step"][t] + (origin if t else 0.0)
        for i in (1, 2):
            x = P.one_layer(x, w, i, raw)
    x = P.one_layer(x, w, 3, raw)
    layers = []
    got = P.logits_of_sequence(raw, w, tokens, layers)
    assert len(layers) == 6 and torch.allclose(layers[-1], x)
    assert torch.allclose(got, P.layer_norm(x, w["final.norm"], w["final.norm.b"], 1e-5) @ w["head"].T)
    assert math.isfinite(got.abs().max().item())
