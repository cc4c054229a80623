"""Bilipel on the GPU against the plain implementation (`plain_bilipel.py`): every mechanism's kernel alone, then whole models of
several small shapes through `bin/trace_run` in every cutting (whole, a decoded tail, portions down to two tokens, requests mixed
in a pool so small that pages and state slots are used again), in float32 and bfloat16, and greedy generation through the engine's
entry point and scheduler.  Where random weights would hide a fault (a far key, a sink, a window's edge, an old token in a recurrent
state), inputs are made so that it shows.

Routing in whole models: in float32 the router chooses freely (the engine's float32 logits and the plain implementation's agree but
for ties); in bfloat16 the layers choose all their experts, so that no close call decides a row."""
import copy
import functools
import json
import os

import pytest
import torch

import plain_bilipel as P
import trace_tools as T

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def gla(heads, dim, vdim, tau, rank):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "decay_rank": rank}}


def attention(heads, kv_heads, dim, vdim, dims, base=500.0, scaling=None, scale=None):
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.5 / dim ** 0.5,
                                           "rot": rot}}


def latent(heads, dim, rot_dim, vdim, kv_rank, window, base=300.0, scale=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                                  "scale": scale or 3.0 / (dim + rot_dim) ** 0.5, "mask": {"size": window},
                                                  "rot": {"base": base, "dims": rot_dim}}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


# X: sizes that no tensor-core kernel takes: every per-head size different, odd widths and vocabulary, windows of 19 positions (no
# multiple of the page size 4) and of one, parts of heads rotated, stretched and plain, layers without a feed-forward, thin products
# of 5 and 3, a tau of 1, 2 of 5, 3 of 3 and 1 of 4 experts, three passes over three layers in the middle.
SHAPE_X = {"architecture": "Bilipel", "vocab": 211, "width": 72, "norm": {"eps": 1e-5}, "residual_mult": 0.4,
           "loop": {"start": 1, "stop": 4, "times": 3}, "layers": [
               dict(gla(3, 20, 14, 4.0, 5), mlp=dense(100)),
               dict(attention(6, 2, 20, 12, 10, scaling=(6.0, 40, 8.0, 1.0)), mlp=moe(5, 2, 20)),
               dict(latent(3, 10, 6, 14, 18, 19), mlp=None),
               dict(gla(1, 6, 10, 1.0, 3), mlp=moe(3, 3, 12)),
               dict(attention(3, 3, 9, 28, 4), mlp=dense(44)),
               dict(latent(2, 8, 2, 8, 40, 1), mlp=moe(4, 1, 16))]}
# Y: sizes of the tensor-core kernels, values that a model may happen to make equal or 1: one pass of a loop over every layer, a
# multiplier of 1, a factor of 1, one expert, one key head for 16 query heads, windows of the page size and longer than any request,
# 32 latent heads (more than a tile of few rows holds), a head rotated whole.
SHAPE_Y = {"architecture": "Bilipel", "vocab": 97, "width": 64, "norm": {"eps": 1e-6}, "residual_mult": 1.0,
           "loop": {"start": 0, "stop": 6, "times": 1}, "layers": [
               dict(gla(2, 16, 16, 16.0, 8), mlp=dense(64)),
               dict(attention(16, 1, 64, 64, 64, scaling=(1.0, 64, 32.0, 1.0)), mlp=moe(1, 1, 64)),
               dict(latent(32, 16, 16, 16, 48, 16), mlp=moe(8, 2, 16)),
               dict(attention(2, 1, 128, 64, 32, scaling=(4.0, 100, 4.0, 1.0)), mlp=None),
               dict(gla(3, 64, 48, 12.0, 8), mlp=dense(128)),
               dict(latent(4, 32, 16, 48, 80, 1000), mlp=moe(4, 2, 64))]}
# Z: no loop and no multiplier (what a file may leave out), heads of 80, 112, 130 and 260 elements, 48 latent heads; W: the same with
# three passes over the last two layers.
SHAPE_Z = {"architecture": "Bilipel", "vocab": 131, "width": 96, "norm": {"eps": 1e-5}, "layers": [
    dict(attention(4, 2, 80, 112, 48, scaling=(8.0, 64, 16.0, 0.5)), mlp=moe(4, 1, 32)),
    dict(gla(2, 130, 70, 8.0, 4), mlp=dense(160)),
    dict(latent(48, 16, 32, 32, 80, 33), mlp=moe(6, 2, 24)),
    dict(gla(1, 260, 24, 16.0, 16), mlp=None)]}
SHAPE_W = dict(copy.deepcopy(SHAPE_Z), loop={"start": 2, "stop": 4, "times": 3}, residual_mult=0.6)
# V: heads of 64 and 128 of equal key and value sizes, windows whose passed pages go back to the pool while a request runs.
SHAPE_V = {"architecture": "Bilipel", "vocab": 151, "width": 128, "norm": {"eps": 1e-6}, "residual_mult": 0.5,
           "loop": {"start": 0, "stop": 2, "times": 2}, "layers": [
               dict(attention(4, 2, 64, 64, 32, scaling=(4.0, 100, 16.0, 1.0)), mlp=dense(192)),
               dict(latent(16, 64, 32, 64, 128, 24), mlp=moe(4, 2, 64)),
               dict(attention(4, 1, 128, 128, 128, base=1e5), mlp=dense(64)),
               dict(gla(2, 64, 128, 16.0, 16), mlp=moe(4, 2, 64))]}
SHAPES = {"X": (SHAPE_X, 4), "Y": (SHAPE_Y, 16), "Z": (SHAPE_Z, 16), "W": (SHAPE_W, 8), "V": (SHAPE_V, 16)}
LENGTHS = {"X": [70, 45, 33, 100, 330, 64, 37, 90], "Y": [1, 7, 17, 40, 129, 65, 96, 290], "Z": [40, 75, 23, 58, 66, 31],
           "W": [50, 2, 81, 64, 33, 47], "V": [150, 40, 97, 300, 64, 130]}
MODES = ("whole", "decode_tail", "portions", "mixed")


def choosing_all(raw):
    """The same model with every routed layer choosing all its experts (for bfloat16: no close calls)."""
    out = copy.deepcopy(raw)
    for layer in out["layers"]:
        if layer["mlp"] is not None and layer["mlp"]["kind"] == "moe":
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return out


def write_model(folder, raw, seed):
    """A seeded random model: its attentions sharpened, its sinks and its routers' logits spread, recurrences that remember dozens
    of tokens with decays that differ from token to token, and one channel that forgets all at once."""
    from mini_rsglang_b200.models import config_from_dict
    from mini_rsglang_b200.weights import write_random_model, write_safetensors
    from mini_rsglang_b200.weights.safetensors_io import SafetensorsFile

    write_random_model(folder, config_from_dict(raw), seed=seed, dtype=torch.bfloat16)
    path = os.path.join(folder, "model.safetensors")
    tensors = {k: t.read() for k, t in SafetensorsFile(path).tensors.items()}
    factors = {"q": 6.0, "k": 6.0, "v": 6.0, "a1": 6.0, "a2": 20.0, "g": 2.5, "uk": 4.0, "uv": 6.0, "dkv": 4.0, "sink": 4.0}
    for name, t in tensors.items():
        leaf = name.split(".")[-1]
        if ".mix." in name and leaf in factors:
            tensors[name] = (t.float() * factors[leaf]).to(t.dtype)
        elif name.endswith("a2.b"):
            bias = t.float() + 2.0
            bias[1] = -60.0
            tensors[name] = bias.to(t.dtype)
        elif name.endswith(".mix.q.norm"):
            tensors[name] = (t.float() * 1.5).to(t.dtype)
        elif name.endswith(".mlp.router"):
            tensors[name] = (t.float() * 12.0).to(t.dtype)
        elif name == "embed":
            tensors[name] = (t.float() * 20.0).to(t.dtype)
    write_safetensors(path, tensors)
    return folder


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for i, (name, (raw, _)) in enumerate(SHAPES.items()):
        out[(name, "float32")] = write_model(str(tmp_path_factory.mktemp(f"bilipel_{name}")), raw, 41 + i)
        out[(name, "bfloat16")] = write_model(str(tmp_path_factory.mktemp(f"bilipel_{name}_all")), choosing_all(raw), 41 + i)
    return out


@functools.lru_cache(maxsize=None)
def plain_logits(folder, name):
    config, weights = P.load(folder)
    reqs = T.requests_for(config["vocab"], LENGTHS[name], seed=300 + ord(name))
    return reqs, {r: P.logits_of_sequence(config, weights, tokens) for r, tokens in reqs.items()}


_results = {}


def replay(folders, name, dtype, tmp_path_factory):
    key = (name, dtype)
    if key in _results:
        return _results[key]
    folder = folders[key]
    reqs, want = plain_logits(folder, name)
    raw, page = SHAPES[name]
    mixed, peak = T.trace_mixed(reqs, seed=9)
    traces = {"whole": T.trace_whole(reqs), "decode_tail": T.trace_decode_tail(reqs, tail=40),
              "portions": T.trace_portions(reqs, seed=6), "mixed": mixed}
    max_tokens = max(peak, max(T.rounded(len(t)) for t in reqs.values()))
    assert sum(T.rounded(len(t)) for t in reqs.values()) > max_tokens, "the pool must force pages to be used again"
    run = T.TraceRun(folder, dtype, str(tmp_path_factory.mktemp(f"out_{name}_{dtype}")), max_tokens, extra=("--page-size", str(page)))
    out, first = {}, 0
    for mode in MODES:
        trace = T.renumber(traces[mode], first, f"{mode}-")
        first += len(trace.steps)
        rows = []
        for step, places in zip(trace.steps, trace.rows):
            got = run.step(step, raw["vocab"])
            if places:
                rows.append((step["step"], got, torch.stack([want[r][p] for r, p in places]), places))
        out[mode] = rows
    assert run.close() == 0
    _results[key] = out
    return out


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SHAPES))
def test_replay_matches_plain(folders, tmp_path_factory, name, dtype, mode):
    """Prefill against token-by-token decoding, portions of every size, batches against each request alone, pages and state slots
    used again; prompts of about 300 tokens take the recurrence in chunks."""
    rows = replay(folders, name, dtype, tmp_path_factory)[mode]
    assert rows
    for step, got, want, _ in rows:
        T.check_rows(got, want, dtype, f"{name} {dtype} {mode} step {step}")


@pytest.mark.parametrize("name", sorted(SHAPES))
def test_float32_logits_do_not_depend_on_the_cutting(folders, tmp_path_factory, name):
    result = replay(folders, name, "float32", tmp_path_factory)
    whole = {place: row for _, got, _, places in result["whole"] for row, place in zip(got, places)}
    compared = 0
    for mode in MODES[1:]:
        for step, got, _, places in result[mode]:
            for row, place in zip(got, places):
                assert (row - whole[place]).abs().max() <= 2e-5 * max(1.0, whole[place].abs().max().item()), (mode, step, place)
                compared += 1
    assert compared > 50


def test_a_prompt_of_more_rows_than_a_recorded_step_holds(tmp_path_factory):
    """2,100 tokens in one step: queued kernel by kernel, the feed-forward's first product from the kernel for many rows, the
    recurrence in many chunks; then decoded tokens from the states that it left."""
    raw = {"architecture": "Bilipel", "vocab": 97, "width": 64, "norm": {"eps": 1e-5}, "residual_mult": 0.5,
           "loop": {"start": 0, "stop": 1, "times": 2}, "layers": [
               dict(gla(2, 16, 32, 16.0, 8), mlp=dense(128)), dict(attention(2, 1, 32, 32, 16, scaling=(5.0, 300, 16.0, 1.0)), mlp=moe(3, 3, 64)),
               dict(latent(4, 16, 16, 16, 32, 70), mlp=dense(64))]}
    folder = write_model(str(tmp_path_factory.mktemp("bilipel_long")), raw, 61)
    config, weights = P.load(folder)
    tokens = T.requests_for(raw["vocab"], [2112], seed=12)["r0"]
    want = P.logits_of_sequence(config, weights, tokens)
    run = T.TraceRun(folder, "bfloat16", str(tmp_path_factory.mktemp("out_long")), T.rounded(2112),
                     env=dict(os.environ, MRS_GEMM_GATED_ROWS_MIN="2048"), extra=("--page-size", "16"))
    got = run.step({"step": 0, "entries": [{"id": "a", "tokens": tokens[:2100], "want": list(range(2100))}], "end": []}, raw["vocab"])
    T.check_rows(got, want[:2100], "bfloat16", "a prompt of 2,100 tokens")
    for t in range(2100, 2112):
        got = run.step({"step": t, "entries": [{"id": "a", "tokens": [tokens[t]], "want": [0]}], "end": []}, raw["vocab"])
        T.check_rows(got, want[t:t + 1], "bfloat16", f"decoded token {t}")
    assert run.close() == 0


# ----------------------------------------------------------------------------------------------------------------
# each mechanism alone
# ----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("width", [72, 320, 1001, 4100, 16500])
def test_layer_norm_adds_a_scaled_branch_a_second_one_and_a_row(width):
    from mini_rsglang_b200 import kernels

    torch.manual_seed(width)
    stream, extra = torch.randn(9, width, device=DEV) * 3, torch.randn(9, width, device=DEV) * 2
    row, weight, bias = (torch.randn(width, device=DEV) for _ in range(3))
    rows = torch.tensor([7, 0, 3], dtype=torch.int32, device=DEV)
    for dtype, tol in ((torch.float32, 3e-6), (torch.bfloat16, 8e-3)):
        for delta_type in {torch.float32, dtype}:
            delta = (torch.randn(9, width, device=DEV) * 4).to(delta_type)
            for parts in range(8):
                total = stream.double().cpu()
                given = {}
                if parts & 1:
                    total = total + 0.3 * delta.double().cpu()
                if parts & 2:
                    total, given["extra"] = total + extra.double().cpu(), extra
                if parts & 4:
                    total, given["row"] = total + row.double().cpu(), row
                want = P.layer_norm(total, weight.double().cpu(), bias.double().cpu(), 1e-5)
                for write_back in (True, False):
                    s, out = stream.clone(), torch.empty(9, width, dtype=dtype, device=DEV)
                    kernels.add_layernorm(s, delta if parts & 1 else None, weight, bias, 1e-5, out, None, write_back, factor=0.3, **given)
                    assert (out.double().cpu() - want).abs().max() < tol * want.abs().max()
                    if write_back:
                        assert (s.double().cpu() - total).abs().max() < 1e-6 * total.abs().max()
                    else:
                        assert torch.equal(s, stream)
                picked = torch.empty(3, width, dtype=dtype, device=DEV)
                kernels.add_layernorm(stream, delta if parts & 1 else None, weight, bias, 1e-5, picked, rows, False, factor=0.3, **given)
                assert (picked.double().cpu() - want[rows.cpu().long()]).abs().max() < tol * want.abs().max()


def test_every_norm_takes_what_is_still_to_be_added():
    """A sum of branches with factors and a vector of the pass, as the stream entry makes it, through a layer norm, an RMS norm and a
    pair of them; nothing is written where the stream must stay."""
    from mini_rsglang_b200.parts.base import NORMS, STREAM_ENTRIES, BranchSum, PartSpec, Runtime
    from mini_rsglang_b200.parts.norm import NormPair

    torch.manual_seed(5)
    width, rows = 40, 7
    runtime = Runtime(torch.device(DEV), torch.float32, 4)
    stream, origin, a, b = (torch.randn(rows, width, device=DEV) for _ in range(4))
    steps = torch.randn(3, width, device=DEV)
    weight, bias = torch.rand(width, device=DEV) + 0.5, torch.randn(width, device=DEV)
    entries = [STREAM_ENTRIES.build(PartSpec("add_embedding_and_step", {"width": width, "times": 3, "number": t, "with_embedding": t > 0, "leaf": ""}),
                                    "s") for t in range(3)]
    assert [len(e.weight_specs()) for e in entries] == [1, 0, 0] and [e.reads_origin for e in entries] == [False, True, True]
    layer = NORMS.build(PartSpec("layernorm", {"width": width, "eps": 1e-5}), "n")
    rms = NORMS.build(PartSpec("rmsnorm", {"width": width, "eps": 1e-5}), "n")
    for part in (*entries, layer, rms):
        part.bind({"s": steps, "n.weight": weight, "n.bias": bias}, runtime)
    for t, entry in enumerate(entries):
        for pending, added in ((None, 0.0), (a, a), (BranchSum([(a, 0.3)]), 0.3 * a), (BranchSum([(a, 0.3), (b, -2.0), (b, 1.0)]), 0.3 * a - b)):
            total = (stream + added + (origin if t else 0.0) + steps[t]).double().cpu()
            joined = entry.join(pending, origin if t else None)
            assert torch.allclose(joined.add_to(stream).double().cpu(), total, atol=2e-6)
            wants = {layer: P.layer_norm(total, weight.double().cpu(), bias.double().cpu(), 1e-5), rms: P.rms_norm(total, weight.double().cpu(), 1e-5)}
            for norm, want in wants.items():
                for write_back in (True, False):
                    s = stream.clone()
                    assert torch.allclose(norm.add_norm(s, joined, write_back=write_back).double().cpu(), want, atol=1e-5)
                    assert torch.allclose(s.double().cpu(), total, atol=2e-6) if write_back else torch.equal(s, stream)
            pair = NormPair(rms, rms)
            s = stream.clone()
            for out in pair.add_norm(s, joined):
                assert torch.allclose(out.double().cpu(), wants[rms], atol=1e-5)


@pytest.mark.parametrize("experts,top,spread", [(5, 2, 3.0), (1, 1, 1.0), (12, 12, 2.0), (70, 40, 3.0), (8, 1, 60.0)])
def test_router_with_a_bias_weighs_the_chosen_logits_alone(experts, top, spread):
    from mini_rsglang_b200 import kernels

    torch.manual_seed(experts * 10 + top)
    tokens = 37
    logits, bias = torch.randn(tokens, experts + 3) * spread, torch.randn(experts) * 2 * spread
    chosen = torch.empty(tokens, top, dtype=torch.int32, device=DEV)
    weights = torch.empty(tokens, top, device=DEV)
    kernels.moe_route(logits.to(DEV), None, chosen, weights, None, experts, top, 1.0, bias=bias.to(DEV))
    z = (logits[:, :experts] + bias).double()
    want_chosen, want_weights = P.choose_experts(z, top)
    assert torch.equal(chosen.cpu().long(), want_chosen)
    assert (weights.double().cpu() - want_weights).abs().max() < 1e-5
    assert (P.choose_experts(logits[:, :experts].double(), top)[0] != want_chosen).any() or top == experts == 1, "the bias decides nothing"


@pytest.mark.parametrize("nq,nkv,d,e,dims,scaling,extra", [
    (6, 2, 20, 12, 10, (6.0, 40, 8.0, 1.0), 0), (6, 3, 112, 112, 40, (8.0, 300, 16.0, 1.0), 0), (3, 3, 9, 28, 4, None, 5), (2, 1, 128, 64, 64, (4.0, 64, 4.0, 1.0), 8),
    (16, 1, 200, 40, 100, (2.0, 4096, 32.0, 1.0), 0), (40, 8, 64, 64, 64, None, 0), (1, 1, 4, 4, 0, None, 0)])
def test_norms_over_whole_projections_then_stretched_rotation(nq, nkv, d, e, dims, scaling, extra):
    from mini_rsglang_b200 import kernels
    from mini_rsglang_b200.parts.base import POSITION_ENCODINGS, PartSpec, Runtime

    torch.manual_seed(d)
    tokens, page, pool = 11, 4, 9
    proj = torch.randn(tokens, nq * d + nkv * d + nkv * e + extra) * torch.exp(torch.randn(tokens, 1))
    proj[:, :d] *= 5.0                                       # one head much larger than the others: a norm a head would show
    positions = torch.tensor([0, 1, 2, 3, 63, 64, 65, 900, 7, 8, 300], dtype=torch.int32)
    slots = torch.randperm(pool * page)[:tokens].to(torch.int32)
    slots[5] = -1
    q_norm, k_norm = torch.rand(nq * d) + 0.5, torch.rand(nkv * d) + 0.5
    params = {"rotary_dim": dims, "theta": 500.0}
    f, m = P.plain_frequencies(500.0, dims), 1.0
    if scaling:
        s = dict(zip(("factor", "original", "fast", "slow"), scaling))
        params.update(s)
        f, m = P.stretched_frequencies(500.0, dims, s)

    class Ctx:
        pass

    ctx = Ctx()
    ctx.positions, ctx.shared = positions.to(DEV), {}
    table = None
    if dims:
        part = POSITION_ENCODINGS.build(PartSpec("yarn_rope", params), "p")
        part.bind({}, Runtime(torch.device(DEV), torch.float32, page))
        table = part.rotations(ctx)
        assert part.rotations(ctx) is table
    x = proj.double()
    q = P.rotate_halves(P.rms_norm(x[:, :nq * d], q_norm.double(), 1e-5).view(tokens, nq, d), positions, f, m)
    k = P.rotate_halves(P.rms_norm(x[:, nq * d:(nq + nkv) * d], k_norm.double(), 1e-5).view(tokens, nkv, d), positions, f, m)
    v = x[:, (nq + nkv) * d:(nq + nkv) * d + nkv * e].view(tokens, nkv, e)
    for dtype, tol in ((torch.float32, 4e-4), (torch.bfloat16, 1e-2)):       # float32: angles of hundreds
        q_out = torch.empty(tokens, nq * d, dtype=dtype, device=DEV)
        k_cache = torch.full((pool, nkv, page, d), 7.0, dtype=dtype, device=DEV)
        v_cache = torch.full((pool, nkv, page, e), 7.0, dtype=dtype, device=DEV)
        kernels.qkv_rotary_store(proj.to(DEV), q_out, k_cache, v_cache, slots.to(DEV), nq, nkv, d, e, rotations=table, rotary_dim=dims,
                                 norm_place="whole_before_rotation", q_norm=q_norm.to(DEV), k_norm=k_norm.to(DEV), norm_eps=1e-5)
        top = max(1.0, q.abs().max().item(), k.abs().max().item(), v.abs().max().item())
        near = positions < 100
        assert (q_out.double().cpu().view(tokens, nq, d) - q).abs().max() < tol * top
        assert dtype is torch.bfloat16 or (q_out.double().cpu().view(tokens, nq, d) - q)[near].abs().max() < 4e-5 * top
        for t in range(tokens):
            if slots[t] >= 0:
                p, at = int(slots[t]) // page, int(slots[t]) % page
                assert (k_cache[p, :, at].double().cpu() - k[t]).abs().max() < tol * top
                assert (v_cache[p, :, at].double().cpu() - v[t]).abs().max() < tol * top
        untouched = sorted(set(range(pool * page)) - {int(s) for s in slots if s >= 0})
        assert (k_cache.transpose(1, 2).reshape(pool * page, -1)[untouched] == 7.0).all()


@pytest.mark.parametrize("H,d,r,R,rotary", [(3, 10, 6, 18, 6), (5, 32, 24, 48, 24), (2, 8, 2, 40, 2), (1, 16, 10, 30, 4), (32, 64, 64, 512, 64)])
def test_latent_rows_turned_in_neighbouring_pairs(H, d, r, R, rotary):
    from mini_rsglang_b200 import kernels

    torch.manual_seed(H * 10 + r)
    tokens, page, pool = 9, 4, 9
    proj = torch.randn(tokens, H * (d + r) + R + r)
    positions = torch.tensor([0, 1, 2, 3, 63, 64, 65, 7, 8], dtype=torch.int32)
    slots = torch.randperm(pool * page)[:tokens].to(torch.int32)
    slots[5] = -1
    f, w = P.plain_frequencies(300.0, rotary), torch.rand(R) + 0.5
    x = proj.double()
    q, low = x[:, :H * (d + r)].view(tokens, H, d + r), x[:, H * (d + r):]
    want_q = P.rotate_neighbours(q[..., d:], positions, f)
    want_rows = torch.cat([P.rms_norm(low[:, :R], w.double(), 1e-5), P.rotate_neighbours(low[:, None, R:], positions, f)[:, 0]], dim=1)
    for dtype, tol in ((torch.float32, 4e-5), (torch.bfloat16, 4e-2)):
        q_plain = torch.empty(H, tokens, d, dtype=dtype, device=DEV)
        q_rows = torch.zeros(tokens, H, R + r, dtype=dtype, device=DEV)
        cache = torch.full((pool, 1, page, R + r), 7.0, dtype=dtype, device=DEV)
        kernels.latent_prepare(proj.to(DEV), w.to(DEV), 1e-5, torch.tensor(f).float().to(DEV), 1.0, positions.to(DEV), slots.to(DEV), q_plain, q_rows,
                               cache, None, H, d, r, R, rotary, True, pairing="interleaved")
        assert (q_plain.double().cpu().transpose(0, 1) - q[..., :d]).abs().max() < tol
        assert (q_rows.double().cpu()[..., R:] - want_q).abs().max() < tol
        flat = cache.double().cpu().view(pool * page, R + r)
        for t in range(tokens):
            if slots[t] >= 0:
                assert (flat[slots[t]] - want_rows[t]).abs().max() < tol, t


def steps_of(lengths, cuts):
    """The portions of several sequences, step by step: [(sequence, first token, tokens)] a step."""
    done, out = [0] * len(lengths), []
    for step in range(max(len(c) for c in cuts)):
        batch = []
        for s in range(len(lengths)):
            if step < len(cuts[s]):
                batch.append((s, done[s], cuts[s][step]))
                done[s] += cuts[s][step]
        out.append(batch)
    assert done == list(lengths)
    return out


def step_facts(batch, slots):
    """(positions, seq_of_token, q_start, state_slots) of a step with a padding sequence behind the real ones."""
    starts = [0]
    for _, _, n in batch:
        starts.append(starts[-1] + n)
    positions = torch.cat([torch.arange(first, first + n) for _, first, n in batch]).to(torch.int32).to(DEV)
    seq = torch.cat([torch.full((n,), i) for i, (_, _, n) in enumerate(batch)]).to(torch.int32).to(DEV)
    return positions, seq, torch.tensor(starts + [starts[-1]], dtype=torch.int32, device=DEV), torch.tensor(
        [slots[s] for s, _, _ in batch] + [-1], dtype=torch.int32, device=DEV)


def scan_case(H, d, e, rank, tau, lengths, seed, extremes=False):
    """Random q, k, v and thin products of several sequences, the second matrix and bias, and the plain functions' read-outs."""
    gen = torch.Generator().manual_seed(seed)
    up, bias = (torch.randn(H * d, rank, generator=gen) / rank ** 0.5).bfloat16(), torch.randn(H * d, generator=gen) + 1.0
    data = []
    for n in lengths:
        q, k, v = (torch.randn(n, H, x, generator=gen) for x in (d, d, e))
        k = k / d ** 0.5
        low = torch.randn(n, rank, generator=gen)
        if extremes:                                         # tokens at which everything, or nearly, is forgotten at once
            low[n // 3] = -1000.0 * up.float()[0] / up.float()[0].pow(2).sum()
            low[n // 2:n // 2 + 9] = -40.0 * up.float()[H * d - 1] / up.float()[H * d - 1].pow(2).sum()
        z = low.double() @ up.double().T + bias.double()
        alpha = torch.exp(P.log_sigmoid(z) / tau).view(n, H, d)
        o, S = P.gla_recurrence(q.double(), k.double(), v.double(), alpha)
        data.append({"q": q, "k": k, "v": v, "low": low, "o": o.reshape(n, H * e), "S": S})
    return data, up, bias


def run_scan(data, up, bias, tau, H, d, e, lengths, cuts, chunk_len, pad=0, dtype=torch.bfloat16):
    """The kernel over the portions of all sequences in slots that held other contents; (o of every sequence, its last state)."""
    from mini_rsglang_b200 import kernels

    slots = [2, 0]
    state = torch.full((3, pad + H * d * e), 11.0, device=DEV)
    S = state[:, pad:].view(3, H, d, e)
    got = [torch.zeros(n, H * e, dtype=torch.float64) for n in lengths]
    up, bias = up.to(dtype).to(DEV), bias.to(DEV)
    rank = up.shape[1]
    for index, batch in enumerate(steps_of(lengths, cuts)):
        rows = torch.cat([torch.cat([data[s][x][first:first + n].reshape(n, -1) for x in ("q", "k", "v", "low")], dim=1) for s, first, n in batch])
        rows = torch.cat([torch.full((rows.shape[0], pad), 99.0), rows], dim=1).to(DEV).contiguous()
        positions, seq, q_start, slot_of = step_facts(batch, slots)
        o = torch.full((rows.shape[0], H * e), 77.0, device=DEV)
        for write in ((False, True) if index == 1 else (True,)):
            before, mine = state.clone(), rows.clone()
            kernels.channel_scan(mine, pad, pad + H * d, pad + 2 * H * d, pad + 2 * H * d + H * e, up, bias, tau, S, positions, seq, q_start,
                                 slot_of, o, H, d, e, write_state=write, chunk_len=chunk_len)
            assert write or torch.equal(before, state), "a step that keeps nothing wrote the state"
            assert torch.equal(mine[:, :pad], rows[:, :pad]) and torch.equal(mine[:, pad + 2 * H * d:], rows[:, pad + 2 * H * d:])
        at = 0
        for s, first, n in batch:
            got[s][first:first + n] = o[at:at + n].double().cpu()
            at += n
    assert (state[1] == 11.0).all() and (state[:, :pad] == 11.0).all(), "memory that no sequence holds was written"
    assert rank == data[0]["low"].shape[1]
    return got, [S[slots[s]].double().cpu() for s in range(len(lengths))]


SCAN_SIZES = [(3, 20, 14, 5), (1, 6, 10, 3), (2, 16, 33, 16), (2, 32, 64, 16), (1, 24, 1, 1), (2, 64, 48, 7), (1, 130, 70, 4), (2, 128, 256, 16), (1, 256, 40, 33),
              (1, 512, 9, 8), (5, 48, 80, 12), (40, 1, 3, 2)]


@pytest.mark.parametrize("extremes", [False, True])
@pytest.mark.parametrize("chunk_len", [0, 13, 64])
@pytest.mark.parametrize("H,d,e,rank", SCAN_SIZES)
def test_channel_scan_in_portions_with_slots_used_again(H, d, e, rank, chunk_len, extremes):
    """In one go and in chunks (also longer than a portion), over two sequences cut into portions of 1 to 70 tokens that begin
    anywhere in a batch of rows, with decays of nothing and of almost nothing among them."""
    lengths, cuts = [115, 61], [[70, 1, 2, 1, 1, 33, 7], [1, 1, 3, 56]]
    tau = 16.0 if d % 32 == 0 else 1.0
    data, up, bias = scan_case(H, d, e, rank, tau, lengths, 5 * d + e, extremes)
    dtype = torch.float32 if d == 20 else torch.bfloat16
    got, states = run_scan(data, up, bias, tau, H, d, e, lengths, cuts, chunk_len, pad=4 if e % 2 == 0 else 3, dtype=dtype)
    for s in range(2):
        for g, want in ((got[s], data[s]["o"]), (states[s], data[s]["S"])):
            assert torch.isfinite(g).all()
            assert (g - want).abs().max() < 3e-5 * max(1.0, want.abs().max().item()), s


@pytest.mark.parametrize("chunk_len", [0, 104])
def test_the_state_still_holds_a_far_token_in_a_channel_that_does_not_forget(chunk_len):
    """Two early values under keys along two channels, one of which halves with every token: 900 tokens later the one is read back
    to the last digit, the other is gone; in one prompt and after 900 decoded tokens."""
    H, d, e, n = 1, 16, 8, 903
    data, up, bias = scan_case(H, d, e, 1, 1.0, [n], 3)
    up, bias = torch.zeros(H * d, 1).bfloat16(), torch.full((H * d,), 60.0)         # every channel keeps everything ...
    bias[9] = 0.0                                                                    # ... but one
    case = data[0]
    case["k"][:, 0, 5] = case["k"][:, 0, 9] = 0.0
    case["q"][:, 0] = 0.0
    case["k"][1:3, 0] = 0.0
    case["k"][1, 0, 5], case["k"][2, 0, 9] = 1.0, 1.0
    case["q"][n - 2, 0, 5], case["q"][n - 1, 0, 9] = 1.0, 1.0
    for cuts in ([n], [3] + [1] * 900):
        if len(cuts) > 1 and chunk_len:
            continue
        got, _ = run_scan([case, case], up, bias, 1.0, H, d, e, [n, n], [cuts, cuts], chunk_len)
        want = case["v"][1, 0].double()
        assert (got[0][n - 2] - want).abs().max() < 3e-5 * want.abs().max()
        assert got[0][:n - 2].abs().max() == 0.0 and got[0][n - 1].abs().max() < 1e-30


def plain_latent_rows_attention(q_rows, rows, R, scale, window, sink):
    seen = P.seen_in_window(q_rows.shape[0], window)
    return torch.stack([P.softmax_with_sink(q_rows[:, h] @ rows.T * scale, seen, sink[h]) @ rows[:, :R] for h in range(q_rows.shape[1])], dim=1)


def run_latent_rows_attention(dtype, q_rows, rows, R, scale, window, sink, page, kernel, give_back=0):
    """The attention kernels on one sequence whose pages lie scattered in a larger pool.  `kernel`: "simt" (one warp a row), "rows",
    "keys" or "split" (the tensor-core kernel over tiles of 64 rows, of 16 rows, of 16 rows with three CTAs a tile), "few" (a token of
    many heads as several rows of 16 heads).  `give_back`: so many of the first pages are -1 in the table."""
    from mini_rsglang_b200 import kernels

    n, H, row = q_rows.shape
    gen = torch.Generator().manual_seed(n)
    pages = -(-n // page)
    pool = pages + 5
    table = torch.randperm(pool, generator=gen)[:pages].to(torch.int32)
    cache = torch.full((pool, 1, page, row), 7.0, dtype=dtype, device=DEV)
    cache.view(pool * page, row)[torch.tensor([int(table[p // page]) * page + p % page for p in range(n)], device=DEV)] = rows.to(dtype).to(DEV)
    table[:give_back] = -1
    q = q_rows.to(dtype).to(DEV).reshape(n, H * row).contiguous()
    out = torch.empty(n, H * R, dtype=dtype, device=DEV)
    positions = torch.arange(n, dtype=torch.int32, device=DEV)
    table, sink = table.view(1, -1).to(DEV), sink.float().to(DEV)
    if kernel == "simt":
        kernels.attention_biased_simt(q, cache, None, positions, torch.zeros(n, dtype=torch.int32, device=DEV), table, out, H, 1, row, R, scale,
                                      window=window, sink_logits=sink)
    elif kernel == "few":
        m = H // 16
        tiles = torch.tensor([[0, t, 1, 0] for t in range(n * m)], dtype=torch.int32, device=DEV)
        kernels.attention_biased_mma(q.view(n * m, 16 * row), cache, None, positions.repeat_interleave(m), table, tiles, out.view(n * m, 16 * R), 16, 1,
                                     row, R, scale, window=window, narrow=True, splits=2, sink_logits=sink)
    else:
        tokens = (64 if kernel == "rows" else 16) // H
        tiles = torch.tensor([[0, t, min(tokens, n - t), 0] for t in range(0, n, tokens)], dtype=torch.int32, device=DEV)
        kernels.attention_biased_mma(q, cache, None, positions, table, tiles, out, H, 1, row, R, scale, window=window, narrow=kernel != "rows",
                                     splits=3 if kernel == "split" else 1, sink_logits=sink)
    kernels.check_device_errors()
    return out.double().cpu().view(n, H, R)


@pytest.mark.parametrize("kernel", ["simt", "rows", "keys", "split", "few"])
@pytest.mark.parametrize("H,R,r,window,page", [(5, 64, 48, 24, 16), (32, 48, 16, 33, 16), (1, 32, 32, 1, 4), (6, 112, 16, 90, 16), (16, 256, 32, 70, 16), (48, 64, 64, 16, 8)])
def test_latent_attention_with_sinks_that_differ_from_head_to_head(kernel, H, R, r, window, page):
    if (kernel in ("keys", "split") and H > 16) or (kernel == "few" and (H % 16 or H == 16)):
        pytest.skip("tiles of 16 rows hold up to 16 heads; rows of 16 heads want a multiple of them")
    torch.manual_seed(H * 100 + R)
    n = 110
    q_rows, rows = torch.randn(n, H, R + r).bfloat16().double(), torch.randn(n, R + r).bfloat16().double()
    sink = torch.linspace(-3.0, 6.0, H).double()
    want = plain_latent_rows_attention(q_rows, rows, R, 0.7 / (R + r) ** 0.5, window, sink)
    got = run_latent_rows_attention(torch.float32 if kernel == "simt" else torch.bfloat16, q_rows, rows, R, 0.7 / (R + r) ** 0.5, window, sink, page, kernel)
    tol = 2e-5 if kernel == "simt" else 0.02
    assert torch.isfinite(got).all() and (got - want).abs().max() < tol * max(1.0, want.abs().max().item())


@pytest.mark.parametrize("kernel", ["simt", "rows", "keys", "split", "few"])
@pytest.mark.parametrize("window,page,n", [(20, 4, 210), (64, 16, 210), (17, 8, 210), (90, 16, 210), (1, 16, 70)])
def test_latent_attention_sees_exactly_its_window(kernel, window, page, n):
    """The last query's one key stands out: the key just inside the window, just outside it, the query's own, the first ones, keys
    at page and block borders.  Where the key is out of sight the sink takes nearly everything.  Passed pages are given back."""
    H, R, r = (32 if kernel == "few" else 2), 16, 16
    torch.manual_seed(window)
    i = n - 1
    dtype, tol = (torch.float32, 1e-5) if kernel == "simt" else (torch.bfloat16, 0.03)
    first_seen = i - window + 1
    targets = sorted({first_seen, first_seen - 1, i, i - 1, 0, 3, first_seen // page * page, first_seen // page * page - 1,
                      (i // page) * page - 1, (i // page) * page, 63, 64, 127, 128} & set(range(n)))
    earliest = max(first_seen - 31, 0)
    give_back = max(earliest - window + 1, 0) // page
    sink = torch.full((H,), 9.0).double()
    for target in targets:
        q_rows, rows = 0.01 * torch.randn(n, H, R + r).double(), 0.01 * torch.randn(n, R + r).double()
        rows[:, :R] += torch.randn(n, R).double()
        q_rows[..., :R] = 0.0
        direction = torch.randn(r).double()
        direction /= direction.norm()
        q_rows[i, :, R:] = 8.0 * direction
        rows[target, R:] = 8.0 * direction
        q_rows, rows = q_rows.bfloat16().double(), rows.bfloat16().double()
        want = plain_latent_rows_attention(q_rows, rows, R, 1.0, window, sink)
        got = run_latent_rows_attention(dtype, q_rows, rows, R, 1.0, window, sink, page, kernel, give_back)
        seen = first_seen <= target
        assert ((want[i, 0] - rows[target, :R]).abs().max() < 1e-2) == seen and (seen or want[i].abs().max() < 0.1), "the plain implementation itself"
        assert (got[earliest:] - want[earliest:]).abs().max() < tol, f"key {target} (seen: {seen}) with window {window}"


def one_sequence(at, m, table, slots):
    """The context of a step that brings the tokens at .. at + m - 1 of one sequence."""
    from mini_rsglang_b200.engine.context import StepContext
    from mini_rsglang_b200.parts.base import StepFacts

    zeros = torch.zeros(m, dtype=torch.int32, device=DEV)
    return StepContext(num_tokens=m, num_sequences=1, token_ids=None, positions=torch.arange(at, at + m, dtype=torch.int32, device=DEV),
                       seq_of_token=zeros, q_start=torch.tensor([0, m], dtype=torch.int32, device=DEV),
                       context_len=torch.tensor([at + m], dtype=torch.int32, device=DEV), state_slots=zeros[:1].clone(), want_rows=None,
                       block_tables=[table.view(1, -1).to(DEV)], slots=[slots.to(torch.int32).to(DEV)], host_q_start=[0, m], host_start_pos=[at],
                       max_query_len=m, max_context_len=at + m, facts=StepFacts([0, m], [at], at + m))


@pytest.mark.parametrize("H,G,d,e,page", [(6, 2, 20, 12, 4), (4, 2, 64, 64, 16), (8, 1, 32, 48, 16), (6, 2, 112, 112, 16), (2, 1, 128, 128, 16), (8, 2, 128, 64, 8)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_attention_reads_far_keys_page_borders_and_sinks(H, G, d, e, page, dtype):
    """The attention as the engine builds it, on one sequence in portions and decoded tokens: each of some places (the first tokens,
    both sides of page borders, far back) is the only key that answers the queries, whose output is then that place's value; before
    that place the sinks take everything."""
    from mini_rsglang_b200 import kernels
    from mini_rsglang_b200.cache.storage import CacheEntry
    from mini_rsglang_b200.parts.base import MIXERS, PartSpec, Runtime

    torch_dtype = getattr(torch, dtype)
    width, n = 16, 333
    part = MIXERS.build(PartSpec("biased_window_attention", {
        "width": width, "num_heads": H, "num_kv_heads": G, "head_dim": d, "value_dim": e, "scale": 40.0 / d, "sink_logits": True,
        "head_norm_eps": 1e-6, "head_norm_place": "whole_before_rotation",
        "position": PartSpec("yarn_rope", {"theta": 300.0, "rotary_dim": d // 4 * 2, "factor": 4.0, "original": 64.0})}), "a")
    eye = torch.eye(H * e)[:min(width, H * e)]
    o_proj = torch.zeros(width, H * e)
    o_proj[:eye.shape[0]] = eye
    vectors = {"a.q_norm.weight": torch.ones(H * d), "a.k_norm.weight": torch.ones(G * d), "a.sinks": torch.linspace(8.0, 12.0, H)}
    tensors = {"a.q_proj.weight": torch.zeros(H * d, width), "a.k_proj.weight": torch.zeros(G * d, width), "a.v_proj.weight": torch.zeros(G * e, width),
               "a.o_proj.weight": o_proj}
    part.bind({**{k: t.to(torch_dtype).to(DEV) for k, t in tensors.items()}, **{k: t.to(DEV) for k, t in vectors.items()}},
              Runtime(torch.device(DEV), torch_dtype, page))
    pages = -(-n // page)
    gen = torch.Generator().manual_seed(d)
    table = torch.randperm(pages + 3, generator=gen)[:pages].to(torch.int32)
    values = torch.randn(n, G, e, generator=gen).bfloat16().float()
    for place in (0, 1, page - 1, page, 5 * page - 1, 5 * page, 200, 299):
        proj = torch.zeros(n, (H + G) * d + G * e)
        proj[:, d - 1:H * d:d] = 12.0                        # the last element of a head does not turn; normed it is sqrt(d)
        proj[:, H * d + d - 2:(H + G) * d:d] = 12.0          # keys along another element ...
        proj[place, H * d:(H + G) * d] = 0.0
        proj[place, H * d + d - 1:(H + G) * d:d] = 12.0      # ... but one
        proj[:, (H + G) * d:] = values.reshape(n, G * e)
        cache = CacheEntry(group=0, k=torch.full((pages + 3, G, page, d), 7.0, dtype=torch_dtype, device=DEV),
                           v=torch.full((pages + 3, G, page, e), -9.0, dtype=torch_dtype, device=DEV))
        at = 0
        for m in [300, 2, 21] + [1] * 10:
            positions = torch.arange(at, at + m, dtype=torch.int32)
            slots = table.long()[positions.long() // page] * page + positions % page
            ctx = one_sequence(at, m, table, slots)
            out = part.forward_projected(proj[at:at + m].to(DEV).contiguous(), 0, ctx, cache).cpu()
            kernels.check_device_errors()
            first = min(max(place - at, 0), m)
            want = torch.cat([values[place, h // (H // G)] for h in range(H)])[:eye.shape[0]]
            assert first == m or (out[first:, :eye.shape[0]] - want).abs().max() < 0.02, (place, at, m)
            assert first == 0 or out[:first].abs().max() < 0.6 * values.abs().max(), "the sinks take the rest"
            at += m


@pytest.mark.parametrize("d,nq,nkv", [(64, 4, 2), (128, 8, 1), (128, 5, 1), (64, 3, 3)])
def test_attention_kernels_fed_by_bulk_copies_take_sinks(d, nq, nkv):
    """The last tokens of one long sequence: decoded tokens whose keys one CTA walks, CTAs of a cluster share, or CTAs that meet
    through memory; a portion whose entries walk all keys or shares of them.  One head's sink takes nearly everything, another's
    nothing; one row's scores all lie far below its sink, one row's far above."""
    from mini_rsglang_b200 import kernels

    n, rows, page = 1500, 40, 16
    torch.manual_seed(d + nq)
    q, k, v = torch.randn(rows, nq, d), torch.randn(n, nkv, d), torch.randn(n, nkv, d)
    q[3] *= 40.0
    k[:, :, 0] += 3.0
    q[5, :, 0] -= 60.0
    q, k, v = (x.bfloat16().double() for x in (q, k, v))
    sink = torch.linspace(-40.0, 14.0, nq).double()
    scale, pages = 0.5 / d ** 0.5, -(-n // page)
    seen = torch.arange(n)[None, :] <= torch.arange(n - rows, n)[:, None]
    want = torch.stack([P.softmax_with_sink(q[:, h] @ k[:, h // (nq // nkv)].T * scale, seen, sink[h]) @ v[:, h // (nq // nkv)] for h in range(nq)], dim=1)
    table = torch.randperm(pages + 4)[:pages].to(torch.int32)
    index = torch.tensor([int(table[p // page]) * page + p % page for p in range(n)])
    caches = []
    for x in (k, v):
        cache = torch.full((pages + 4, page, nkv, d), 7.0, dtype=torch.bfloat16)
        cache.view(-1, nkv, d)[index] = x.bfloat16()
        caches.append(cache.transpose(1, 2).contiguous().to(DEV))
    dq, positions, dsink = q.bfloat16().reshape(rows, nq * d).to(DEV), torch.arange(n - rows, n, dtype=torch.int32, device=DEV), sink.float().to(DEV)
    table = table.view(1, -1).to(DEV)

    def check(out, what):
        kernels.check_device_errors(certain=True)
        got = out.double().cpu().view(rows, nq, d)
        assert torch.isfinite(got).all() and (got - want).abs().max() < 0.03, (what, (got - want).abs().max())

    single = torch.tensor([[0, t, 1, 0] for t in range(rows)], dtype=torch.int32, device=DEV)
    for splits in (1, 2, 8, 5):
        out = torch.empty(rows, nq * d, dtype=torch.bfloat16, device=DEV)
        kernels.attention_decode_tma(dq, *caches, positions, table, single, out, nq, nkv, d, splits=splits, scale=scale, sink_logits=dsink)
        check(out, f"{splits} shares")
    for entries in ([[0, 0, rows, 0]], [[0, 0, rows, s | 3 << 8] for s in range(3)]):
        if rows * (nq // nkv) > 2 * (128 // (nq // nkv)) * (nq // nkv):
            half = 128 // (nq // nkv)
            entries = [[0, at, min(2 * half, rows - at), e[3]] for at in range(0, rows, 2 * half) for e in entries]
        out = torch.empty(rows, nq * d, dtype=torch.bfloat16, device=DEV)
        kernels.attention_prefill_tc(dq, *caches, positions, table, torch.tensor(entries, dtype=torch.int32, device=DEV), out, nq, nkv, d,
                                     scale=scale, shares=entries[0][3] != 0, sink_logits=dsink)
        check(out, entries)


@pytest.mark.parametrize("rows,inner,width", [(1, 128, 72), (13, 192, 136), (300, 64, 64), (2100, 320, 200)])
def test_gelu_gate_in_the_products_and_alone(rows, inner, width):
    from mini_rsglang_b200 import kernels

    torch.manual_seed(rows)
    x = torch.randn(rows, width).bfloat16()
    gate, up = (torch.randn(inner, width).bfloat16() * 0.3 for _ in range(2))
    g, u = x.double() @ gate.double().T, x.double() @ up.double().T
    want = P.gelu_tanh(g) * u
    blocked = torch.stack([gate.view(-1, 64, width), up.view(-1, 64, width)], dim=1).reshape(2 * inner, width).contiguous().to(DEV)
    tol = 6e-3 * want.abs().max()
    out = torch.empty(rows, inner, dtype=torch.bfloat16, device=DEV)
    if rows <= 16:
        kernels.gemm_tc(x.to(DEV), blocked, out, gated=True, gate="gelu_tanh")
        assert (out.double().cpu() - want).abs().max() < tol
    out.fill_(0)
    kernels.gemm_gated_rows(x.to(DEV), blocked, out, "gelu_tanh")
    kernels.check_device_errors(certain=True)
    assert (out.double().cpu() - want).abs().max() < tol
    for dtype, limit in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
        z = torch.cat([g, u], dim=1).to(dtype)
        exact = P.gelu_tanh(z[:, :inner].double()) * z[:, inner:].double()
        out = torch.empty(rows, inner, dtype=dtype, device=DEV)
        kernels.gated_activation(z.to(DEV), out, "gelu_tanh")
        assert (out.double().cpu() - exact).abs().max() < limit * exact.abs().max()


def test_the_stream_after_every_layer(folders, tmp_path_factory):
    """`bin/trace_run --observe`: the float32 residual stream after every layer run against the plain implementation, in a prompt's
    portion and in decoded tokens."""
    import numpy as np

    folder = folders[("X", "float32")]
    config, weights = P.load(folder)
    tokens = T.requests_for(config["vocab"], [19], seed=77)["r0"]
    layers = []
    P.logits_of_sequence(config, weights, tokens, layers)
    assert len(layers) == 12
    out = str(tmp_path_factory.mktemp("observed"))
    run = T.TraceRun(folder, "float32", out, 64, extra=("--page-size", "4", "--observe", "a"))
    for step, (at, m) in enumerate(((0, 16), (16, 1), (17, 2))):
        run.step({"step": step, "entries": [{"id": "a", "tokens": tokens[at:at + m], "want": []}], "end": []}, config["vocab"])
        for i, stream in enumerate(layers):
            got = np.fromfile(os.path.join(out, "observe", f"{step}.layer{i}-output.f32"), dtype="<f4").reshape(m, config["width"])
            want = stream[at:at + m]
            assert (torch.from_numpy(got).double() - want).abs().max() < 2e-5 * max(1.0, want.abs().max().item()), (step, i)
    assert run.close() == 0


# ----------------------------------------------------------------------------------------------------------------
# the engine's own entry point and scheduler
# ----------------------------------------------------------------------------------------------------------------
def check_greedy(config, weights, prompt, generated, dtype):
    """Every generated token is the plain implementation's arg-max behind what came before it, or within rounding of it."""
    logits = P.logits_of_sequence(config, weights, list(prompt) + list(generated))
    for i, token in enumerate(generated):
        row = logits[len(prompt) - 1 + i]
        gap = (row.max() - row[token]).item()
        limit = 2e-5 * max(1.0, row.abs().max().item()) if dtype == "float32" else 0.02 * row.abs().max().item()
        assert gap <= limit, f"{dtype}: engine chose {token}, plain {int(row.argmax())}, gap {gap}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["X", "Y", "V"])
def test_greedy_generation_through_the_engine(folders, name, dtype):
    """Prompts of unequal lengths, more requests than run at a time (state slots are used again), prompt portions under a small
    token budget beside decoded tokens, 60 generated tokens each."""
    from mini_rsglang_b200 import RuntimeConfig, SamplingParams
    from mini_rsglang_b200.engine import EngineHandle

    config, weights = P.load(folders[(name, dtype)])
    prompts = [T.requests_for(config["vocab"], [n], seed=500 + n)["r0"] for n in (3, 50, 1, 77, 20, 31)]
    engine = EngineHandle.load(folders[(name, dtype)], 0, dtype=dtype, num_pages=120 if name == "X" else 40,
                               config=RuntimeConfig(max_seq_len=160, prefill_budget=24, max_running=3, page_size=SHAPES[name][1]))
    results = engine.generate_many(prompts, SamplingParams(max_tokens=60, ignore_eos=True))
    engine.shutdown()
    for prompt, result in zip(prompts, results):
        assert len(result.token_ids) == 60
        check_greedy(config, weights, prompt, result.token_ids, dtype)


def test_one_request_at_a_time(folders):
    """An engine with a single state slot."""
    from mini_rsglang_b200 import RuntimeConfig, SamplingParams
    from mini_rsglang_b200.engine import EngineHandle

    folder = folders[("X", "float32")]
    config, weights = P.load(folder)
    engine = EngineHandle.load(folder, 0, config=RuntimeConfig(max_seq_len=64, prefill_budget=64, max_running=1, page_size=4), dtype="float32",
                               num_pages=16)
    prompts = [[5, 9, 2, 200, 17], [8, 8]]
    for prompt, result in zip(prompts, engine.generate_many(prompts, SamplingParams(max_tokens=8, ignore_eos=True))):
        check_greedy(config, weights, prompt, result.token_ids, "float32")
    engine.shutdown()


def test_command_line_generates_the_plain_tokens(folders):
    import subprocess
    import sys

    folder = folders[("X", "float32")]
    prompt = [3, 1, 4, 1, 5, 9, 2, 6]
    cmd = [sys.executable, os.path.join(T.ROOT, "bin", "mini-rsglang"), "--model", folder, "--dtype", "float32", "--page-size", "4",
           "--max-seq-len", "128", "--num-pages", "40", "generate", "--token-ids", ",".join(map(str, prompt)), "--max-tokens", "12",
           "--ignore-eos", "--json"]
    proc = subprocess.run(cmd, capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr
    events = [json.loads(line) for line in proc.stdout.splitlines() if line.startswith("{")]
    tokens = [e["Token"]["token_id"] for e in events if "Token" in e]
    assert events[-1]["Finished"]["completion_tokens"] == 12 == len(tokens)
    check_greedy(*P.load(folder), prompt, tokens, "float32")
