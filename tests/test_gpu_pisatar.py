"""Pisatar on the GPU against the plain implementation (`plain_pisatar.py`): every mechanism's kernel alone, then whole models
of several small shapes through `bin/trace_run` in every cutting (whole, a decoded tail, portions down to two tokens, requests
mixed in a pool so small that pages and state slots are used again), in float32 and bfloat16, and greedy generation through the
engine's entry point and scheduler.  Where random weights would hide a fault (a far key, an old token in a recurrent state, a
page border), inputs are made so that it shows."""
import functools
import json
import os

import pytest
import torch

import plain_pisatar as P
import trace_tools as T

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def retention(heads, dim, vdim, decay, base=10000.0, dims=None):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay,
                                           "rot": {"base": base, "dims": dim if dims is None else dims}}}


def channel_delta(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv,
                                               "decay_rank": decay_rank, "gate_rank": gate_rank}}


def both(left, right, cap, scales, scale=None, dims=None, base=10000.0, scaling=None):
    heads, kv_heads, dim, vdim = left
    rot = {"base": base, "dims": dim if dims is None else dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 2.0 / dim ** 0.5, "rot": rot},
        "right": {"heads": right[0], "dim": right[1], "vdim": right[2], "gate_cap": cap}, "left_scale": scales[0], "right_scale": scales[1]}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


# X: sizes that no tensor-core kernel takes: every per-head size different, odd widths and vocabulary, rotated parts that are no
# multiple of 8 or nothing at all, query/key heads shared by two and by three value heads, ranks of 5 and 9, layers without a
# feed-forward, a layer whose weights are used twice more (once through another layer that uses them), a negative factor.
_X0 = dict(channel_delta(4, 2, 24, 12, 3, 5, 9), mlp=dense(100))
_X1 = dict(both((6, 2, 20, 12), (3, 12, 20), 7.0, (0.8, -1.3), dims=10, base=500.0, scaling=(6.0, 1.0, 3.0, 40)), mlp=None)
SHAPE_X = {"architecture": "Pisatar", "vocab": 211, "width": 72, "norm": {"eps": 1e-5}, "layers": [
    _X0, _X1, dict(retention(3, 20, 14, [0.9, 0.99, 1.0], dims=12), mlp=dense(52)),
    dict(_X0, weights_of=0), dict(_X1, weights_of=1), dict(channel_delta(3, 1, 8, 30, 2, 3, 4), mlp=None),
    dict(_X0, weights_of=3), dict(retention(1, 6, 10, [0.5], dims=0), mlp=dense(36))]}
# Y: sizes of the tensor-core kernels, values that a model may happen to make equal or 1: one head, a convolution of one tap, every
# frequency of one band, equal key and value sizes that the
# attention kernels fed by bulk copies take, different ones that they do not, 8 query heads a key head, factors of 1 and 0.
SHAPE_Y = {"architecture": "Pisatar", "vocab": 97, "width": 64, "norm": {"eps": 1e-6}, "layers": [
    dict(both((4, 2, 64, 64), (2, 16, 16), 15.0, (1.0, 1.0), dims=64), mlp=dense(64)),
    dict(channel_delta(1, 1, 16, 16, 1, 8, 8), mlp=dense(48)),
    dict(retention(4, 32, 64, [0.3, 0.9, 0.97, 0.9995]), mlp=None),
    dict(both((8, 1, 32, 48), (1, 32, 64), 2.0, (0.5, 1.0), dims=16, scaling=(4.0, 2.0, 2.0, 64)), mlp=dense(80)),
    dict(channel_delta(4, 4, 32, 32, 4, 16, 16), mlp=dense(128)),
    dict(both((2, 1, 128, 128), (1, 8, 8), 15.0, (1.0, 0.0), base=1e6, scaling=(8.0, 1.0, 4.0, 100000)), mlp=dense(16))]}
SHAPES = {"X": (SHAPE_X, 4), "Y": (SHAPE_Y, 16)}
LENGTHS = {"X": [70, 45, 33, 100, 330, 64, 37, 90], "Y": [1, 7, 17, 40, 129, 65, 96, 290]}
MODES = ("whole", "decode_tail", "portions", "mixed")


def write_model(folder, raw, seed):
    """A seeded random model with sharpened attentions, recurrences that remember dozens of tokens (a state that was lost or
    mixed up shows), and gates, step sizes and decays that differ from token to token."""
    from mini_rsglang_b200.models import config_from_dict
    from mini_rsglang_b200.weights import write_random_model, write_safetensors
    from mini_rsglang_b200.weights.safetensors_io import SafetensorsFile

    write_random_model(folder, config_from_dict(raw), seed=seed, dtype=torch.bfloat16)
    path = os.path.join(folder, "model.safetensors")
    tensors = {k: t.read() for k, t in SafetensorsFile(path).tensors.items()}
    factors = {"q": 6.0, "k": 6.0, "v": 6.0, "b": 8.0, "a1": 6.0, "a2": 20.0, "g1": 6.0, "g2": 20.0, "i": 8.0, "f": 8.0, "g": 6.0}
    for name, t in tensors.items():
        leaf = name.split(".")[-1]
        if ".mix." in name and leaf in factors and t.dim() == 2:
            tensors[name] = (t.float() * factors[leaf]).to(t.dtype)
        elif name.endswith(".A_log"):
            tensors[name] = (t.float() - 2.0).to(t.dtype)
        elif name.endswith(".f.b"):
            tensors[name] = (t.float() + 3.0).to(t.dtype)
        elif name.startswith("embed") and t.dim() == 2:
            tensors[name] = (t.float() * 10.0).to(t.dtype)
        elif t.dim() == 1 and (name.endswith("norm") or "norm" in leaf) and ".mix." not in name:
            tensors[name] = (t.float() * 6.0).to(t.dtype)          # weights far enough from their zero that a lost 1 + w shows
    write_safetensors(path, tensors)
    return folder


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: write_model(str(tmp_path_factory.mktemp(f"pisatar_{name}")), raw, 31 + i) for i, (name, (raw, _)) in enumerate(SHAPES.items())}


def load_plain(folder):
    from mini_rsglang_b200.weights.safetensors_io import SafetensorsFile

    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    return config, {k: t.read() for k, t in SafetensorsFile(os.path.join(folder, "model.safetensors")).tensors.items()}


@functools.lru_cache(maxsize=None)
def plain_logits(folder, name):
    config, weights = load_plain(folder)
    reqs = T.requests_for(config["vocab"], LENGTHS[name], seed=300 + ord(name))
    return reqs, {r: P.forward(config, weights, tokens) for r, tokens in reqs.items()}


_results = {}


def replay(folders, name, dtype, tmp_path_factory):
    key = (name, dtype)
    if key in _results:
        return _results[key]
    folder = folders[name]
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
@pytest.mark.parametrize("name", ["X", "Y"])
def test_replay_matches_plain(folders, tmp_path_factory, name, dtype, mode):
    """Prefill against token-by-token decoding, portions of every size, batches against each request alone, pages and state
    slots used again; prompts of 290 and 330 tokens take the recurrences that are linear in their state in chunks."""
    rows = replay(folders, name, dtype, tmp_path_factory)[mode]
    assert rows
    for step, got, want, _ in rows:
        T.check_rows(got, want, dtype, f"{name} {dtype} {mode} step {step}")


@pytest.mark.parametrize("name", ["X", "Y"])
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
    recurrences in many chunks; then decoded tokens from the states that it left."""
    raw = {"architecture": "Pisatar", "vocab": 97, "width": 64, "norm": {"eps": 1e-5}, "layers": [
        dict(retention(2, 16, 32, [0.99, 0.9995]), mlp=dense(64)),
        dict(both((2, 1, 16, 16), (2, 16, 16), 10.0, (0.7, 0.9), dims=8, scaling=(5.0, 1.0, 3.0, 300)), mlp=dense(96)),
        dict(channel_delta(2, 1, 16, 16, 2, 8, 4), mlp=dense(32))]}
    folder = write_model(str(tmp_path_factory.mktemp("pisatar_long")), raw, 61)
    config, weights = load_plain(folder)
    tokens = T.requests_for(raw["vocab"], [2112], seed=12)["r0"]
    want = P.forward(config, weights, tokens)
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
@pytest.mark.parametrize("width", [72, 320, 1001, 4100, 8200])
def test_sum_of_scaled_branches_and_both_next_norms(width):
    from mini_rsglang_b200 import kernels

    torch.manual_seed(width)
    stream = torch.randn(9, width, device=DEV) * 3
    branches = [(torch.randn(9, width, device=DEV) * s, f) for s, f in ((2.0, 0.6), (5.0, -1.5), (1.0, 1.0))]
    weights = [torch.rand(width, device=DEV) + 0.5 for _ in range(2)]
    for count in (0, 1, 2, 3):
        total = stream.double().cpu() + sum(f * x.double().cpu() for x, f in branches[:count])
        for norms in ((0, 1, 2) if count else (1, 2)):
            for dtype, tol in ((torch.float32, 3e-6), (torch.bfloat16, 8e-3)):
                s = stream.clone()
                outs = [(w, torch.empty(9, width, dtype=dtype, device=DEV)) for w in weights[:norms]]
                kernels.add_scaled_branches_norms(s, branches[:count], outs, 1e-5)
                assert (s.double().cpu() - total).abs().max() < 1e-6 * total.abs().max()
                for w, out in outs:
                    want = P.over_rms(total, 1e-5) * w.double().cpu()
                    assert (out.double().cpu() - want).abs().max() < tol * want.abs().max()


@pytest.mark.parametrize("width", [72, 300, 2049])
def test_normed_embeddings(width):
    from mini_rsglang_b200 import kernels

    torch.manual_seed(width)
    ids = torch.tensor([36, 0, 5, 5, 17], dtype=torch.int32, device=DEV)
    weight = torch.randn(width, device=DEV) + 1.0
    for dtype in (torch.float32, torch.bfloat16):
        table = (torch.randn(37, width, device=DEV) * 0.01).to(dtype)          # small rows: the epsilon counts
        stream = torch.empty(5, width, device=DEV)
        kernels.embed_norm(table, ids, weight, 1e-5, stream)
        want = P.over_rms(table.double().cpu()[ids.cpu().long()], 1e-5) * weight.double().cpu()
        assert (stream.double().cpu() - want).abs().max() < 3e-6 * want.abs().max()


@pytest.mark.parametrize("heads,d,dims,offset,extra", [(4, 32, 32, 0, 0), (6, 20, 10, 4, 3), (3, 24, 16, 8, 0), (2, 64, 24, 4, 4), (5, 6, 2, 1, 0)])
def test_heads_turn_in_place(heads, d, dims, offset, extra):
    from mini_rsglang_b200 import kernels

    torch.manual_seed(d)
    tokens = 9
    rows = torch.randn(tokens, offset + heads * d + extra)
    positions = torch.tensor([0, 1, 2, 77, 78, 1000, 5, 4095, 3], dtype=torch.int32)
    f = P.plain_frequencies({"base": 500.0, "dims": dims})
    dev = rows.to(DEV)
    table = kernels.rotation_table(positions.to(DEV), torch.tensor(f, dtype=torch.float64).float().to(DEV))
    kernels.rotate_heads_(dev, offset, heads, d, table, dims)
    want = rows.double().clone()
    want[:, offset:offset + heads * d] = P.rotate(rows.double()[:, offset:offset + heads * d].reshape(tokens, heads, d), f, positions).reshape(tokens, -1)
    assert (dev.double().cpu() - want).abs().max() < 1.5e-3          # angles of thousands in float32
    near = positions < 100
    assert (dev.double().cpu() - want)[near].abs().max() < 3e-5


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
    """(positions, q_start, state_slots) of a step with a padding sequence behind the real ones."""
    starts = [0]
    for _, _, n in batch:
        starts.append(starts[-1] + n)
    positions = torch.cat([torch.arange(first, first + n) for _, first, n in batch]).to(torch.int32).to(DEV)
    return positions, torch.tensor(starts + [starts[-1]], dtype=torch.int32, device=DEV), torch.tensor(
        [slots[s] for s, _, _ in batch] + [-1], dtype=torch.int32, device=DEV)


@pytest.mark.parametrize("cap,heads", [(15.0, 4), (2.0, 1), (40.0, 3)])
def test_gates_of_an_exponential_memory(cap, heads):
    """Raw gates far into the caps, biases, the running maximum from zero, over portions of 1 to 700 tokens (more than a block's
    worth at a time), in slots that held other maxima."""
    from mini_rsglang_b200 import kernels

    torch.manual_seed(int(cap))
    lengths, cuts = [760, 61], [[700, 1, 2, 57], [1, 1, 3, 56]]
    raw = [torch.randn(n, 2 * heads + 3) * 8 - torch.tensor([0.0] * (heads + 1) + [6.0] * (heads + 2)) for n in lengths]
    bias_i, bias_f = torch.randn(heads), torch.randn(heads) + 2
    want = []
    for r in raw:
        log_in = P.capped(r[:, 1:1 + heads].double() + bias_i.double(), cap)
        log_keep = P.log_sigmoid(P.capped(r[:, 2 + heads:2 + 2 * heads].double() + bias_f.double(), cap))
        m, rows = torch.zeros(heads, dtype=torch.float64), []
        for t in range(r.shape[0]):
            top = torch.maximum(log_keep[t] + m, log_in[t])
            rows.append(torch.cat([torch.exp(log_keep[t] + m - top), torch.exp(log_in[t] - top), torch.exp(-top)]))
            m = top
        want.append(torch.stack(rows))
    state = torch.full((3, heads + 5), 9.0, device=DEV)
    got = [torch.zeros(n, 3 * heads, dtype=torch.float64) for n in lengths]
    for index, batch in enumerate(steps_of(lengths, cuts)):
        rows = torch.cat([raw[s][first:first + n] for s, first, n in batch]).to(DEV).contiguous()
        positions, q_start, slots = step_facts(batch, [2, 0])
        coef = torch.empty(rows.shape[0], 3 * heads, device=DEV)
        for write in ((False, True) if index == 1 else (True,)):
            before = state.clone()
            kernels.memory_gates(rows, 1, 2 + heads, bias_i.to(DEV), bias_f.to(DEV), cap, state[:, 5:], positions, q_start, slots, coef, write)
            assert write or torch.equal(before, state)
        at = 0
        for s, first, n in batch:
            got[s][first:first + n] = coef[at:at + n].double().cpu()
            at += n
    for s in range(2):
        assert torch.allclose(got[s], want[s], rtol=3e-5, atol=1e-7), (got[s] - want[s]).abs().max()
    assert (state[1] == 9.0).all() and (state[:, :5] == 9.0).all()


def scan_case(H, d, e, lengths, seed, decay=None, extremes=False):
    """Random q, k, v (and keep, take) of several sequences and the plain functions' read-outs."""
    gen = torch.Generator().manual_seed(seed)
    data = []
    for n in lengths:
        q, k, v = (torch.randn(n, H, x, generator=gen) for x in (d, d, e))
        k = k / d ** 0.5
        keep = torch.rand(n, H, generator=gen) * 0.2 + 0.8
        take = torch.rand(n, H, generator=gen)
        if extremes:
            keep[n // 3] = 1e-7
            keep[n // 2:n // 2 + 9] = 1e-3
            keep[2 * n // 3] = 0.0
            take[n // 4] = 0.0
        o, c = torch.empty(n, H, e, dtype=torch.float64), torch.empty(n, H, dtype=torch.float64)
        for h in range(H):
            S, norm = torch.zeros(d, e, dtype=torch.float64), torch.zeros(d, dtype=torch.float64)
            for t in range(n):
                a, b = (decay[h], 1.0) if decay is not None else (keep[t, h].double(), take[t, h].double())
                S = a * S + b * torch.outer(k[t, h].double(), v[t, h].double())
                norm = a * norm + b * k[t, h].double()
                o[t, h], c[t, h] = S.T @ q[t, h].double(), norm @ q[t, h].double()
        data.append({"q": q, "k": k, "v": v, "coef": torch.cat([keep, take, torch.zeros(n, H)], dim=1), "o": o.reshape(n, H * e), "c": c})
    return data


def run_scan(data, H, d, e, lengths, cuts, decay, normaliser, chunk_len, pad=0):
    """The kernel over the portions of all sequences in slots that held other contents; (o, c) of every sequence."""
    from mini_rsglang_b200 import kernels

    slots = [2, 0]
    state = torch.full((3, pad + H * (d * e + d)), 11.0, device=DEV)
    S, n_state = state[:, pad:pad + H * d * e].view(3, H, d, e), state[:, pad + H * d * e:].view(3, H, d)
    got = [(torch.zeros(n, H * e, dtype=torch.float64), torch.zeros(n, H, dtype=torch.float64)) for n in lengths]
    for index, batch in enumerate(steps_of(lengths, cuts)):
        rows = torch.cat([torch.cat([data[s][x][first:first + n].reshape(n, -1) for x in ("q", "k", "v")], dim=1) for s, first, n in batch])
        rows = torch.cat([torch.full((rows.shape[0], pad), 99.0), rows], dim=1).to(DEV).contiguous()
        coef = torch.cat([data[s]["coef"][first:first + n] for s, first, n in batch]).to(DEV).contiguous()
        positions, q_start, slot_of = step_facts(batch, slots)
        o = torch.full((rows.shape[0], H * e), 77.0, device=DEV)
        c = torch.full((rows.shape[0], H), 77.0, device=DEV)
        for write in ((False, True) if index == 1 else (True,)):
            before = state.clone()
            kernels.linear_scan(rows, pad, pad + H * d, pad + 2 * H * d, torch.tensor(decay, device=DEV) if decay is not None else None,
                                None if decay is not None else coef, S, n_state if normaliser else None, positions, q_start, slot_of, o,
                                c if normaliser else None, H, d, e, write_state=write, chunk_len=chunk_len)
            assert write or torch.equal(before, state), "a step that keeps nothing wrote the state"
        at = 0
        for s, first, n in batch:
            got[s][0][first:first + n] = o[at:at + n].double().cpu()
            got[s][1][first:first + n] = c[at:at + n].double().cpu()
            at += n
    assert (state[1] == 11.0).all() and (state[:, :pad] == 11.0).all(), "memory that no sequence holds was written"
    assert normaliser or (n_state == 11.0).all()
    return got


SCAN_SIZES = [(3, 20, 14), (1, 6, 10), (2, 16, 33), (2, 32, 64), (1, 24, 1), (2, 64, 48), (1, 130, 70), (2, 128, 256), (1, 256, 40), (1, 512, 9)]


@pytest.mark.parametrize("chunk_len", [0, 13, 64])
@pytest.mark.parametrize("H,d,e", SCAN_SIZES)
def test_linear_scan_in_portions_with_slots_used_again(H, d, e, chunk_len):
    """Gates a token with a normaliser, in one go and in chunks (also longer than a portion), over two sequences cut into
    portions of 1 to 70 tokens, with keeps of zero and of almost nothing among them."""
    lengths, cuts = [115, 61], [[70, 1, 2, 1, 1, 33, 7], [1, 1, 3, 56]]
    data = scan_case(H, d, e, lengths, 5 * d + e, extremes=True)
    got = run_scan(data, H, d, e, lengths, cuts, None, True, chunk_len, pad=4 if e % 2 == 0 else 3)
    for s in range(2):
        for i, key in enumerate(("o", "c")):
            want = data[s][key]
            assert (got[s][i] - want).abs().max() < 3e-5 * max(1.0, want.abs().max().item()), (s, key)


@pytest.mark.parametrize("chunk_len", [0, 40])
@pytest.mark.parametrize("H,d,e", SCAN_SIZES)
def test_linear_scan_with_a_constant_decay(H, d, e, chunk_len):
    decay = [0.97, 0.0, 0.002][:H] if d != 32 else [0.9995, 1.0]
    lengths, cuts = [115, 61], [[70, 1, 2, 1, 1, 33, 7], [1, 1, 3, 56]]
    data = scan_case(H, d, e, lengths, 7 * d + e, decay=decay)
    got = run_scan(data, H, d, e, lengths, cuts, decay, False, chunk_len)
    for s in range(2):
        want = data[s]["o"]
        assert (got[s][0] - want).abs().max() < 3e-5 * max(1.0, want.abs().max().item()), s


@pytest.mark.parametrize("chunk_len", [0, 100])
def test_a_retention_still_holds_a_far_token(chunk_len):
    """One early token's value under a key that no other token has, read 900 tokens later through a slow decay: in the float32
    state it is there to the last digit that the decay leaves, in one prompt and after 900 decoded tokens."""
    H, d, e, n, decay = 1, 16, 8, 903, [0.999]
    data = scan_case(H, d, e, [n], 3, decay=decay)[0]
    data["k"][:, 0, 5] = 0.0
    data["q"][:, 0] = 0.0
    data["k"][2, 0] = 0.0
    data["k"][2, 0, 5] = 1.0
    data["q"][n - 1, 0, 5] = 1.0
    want = data["v"][2, 0].double() * 0.999 ** (n - 3)
    for cuts in ([n], [3] + [1] * 900):
        if len(cuts) > 1 and chunk_len:
            continue
        data["o"] = torch.zeros(n, H * e)
        got = run_scan([data, data], H, d, e, [n, n], [cuts, cuts], decay, False, chunk_len)
        assert (got[0][0][n - 1] - want).abs().max() < 3e-5 * want.abs().max()
        assert got[0][0][:n - 1].abs().max() == 0.0


@pytest.mark.parametrize("H,e", [(3, 20), (2, 64), (4, 70), (1, 1), (2, 128), (2, 256), (1, 512), (1, 600)])
def test_head_norm_with_gate_weights_and_normaliser(H, e):
    from mini_rsglang_b200 import kernels

    torch.manual_seed(e)
    tokens = 13
    o, wide = torch.randn(tokens, H * e) * 0.05, torch.randn(tokens, 8 + H * e + 4)
    gate = wide[:, 8:8 + H * e]
    c, floor = torch.randn(tokens, H) * 3, torch.rand(tokens, 3 * H + 1)
    floor_columns = floor[:, 2 * H:3 * H]
    gates = {"silu": P.silu(gate.double()), "sigmoid": torch.sigmoid(gate.double())}
    for kind in gates:
        for weight in (None, torch.rand(e) + 0.5, torch.rand(H * e) + 0.5):
            for normaliser in (None, 1e-6):
                factor = 0.3
                x = o.double().view(tokens, H, e) * factor
                if normaliser:
                    x = x / (torch.maximum((c.double() * factor).abs(), floor_columns.double()) + normaliser)[:, :, None]
                y = P.over_rms(x, 1e-3)
                y = y.reshape(tokens, H * e) if weight is None else (y.reshape(tokens, H * e) * (weight.double() if weight.numel() == H * e
                                                                                                  else weight.double().repeat(H)))
                want = y * gates[kind]
                for dtype, tol in ((torch.float32, 5e-6), (torch.bfloat16, 8e-3)):
                    out = torch.empty(tokens, H * e, dtype=dtype, device=DEV)
                    kernels.head_norm_gate(o.to(DEV), wide.to(DEV)[:, 8:8 + H * e], weight.to(DEV) if weight is not None else None, 1e-3, out, H,
                                           gate_kind=kind, factor=factor,
                                           normaliser=(c.to(DEV), floor.to(DEV)[:, 2 * H:3 * H], normaliser) if normaliser else None)
                    assert (out.double().cpu() - want).abs().max() < tol * max(want.abs().max().item(), 1e-3)


def test_narrowed_columns():
    from mini_rsglang_b200 import kernels

    rows = torch.randn(7, 30, device=DEV)
    for dtype in (torch.float32, torch.bfloat16):
        out = torch.full((7, 16), 5.0, dtype=dtype, device=DEV)
        kernels.narrow_columns(rows, 11, 14, out)
        assert torch.equal(out[:, :14], rows[:, 11:25].to(dtype)) and (out[:, 14:] == 0).all()


@pytest.mark.parametrize("H,G,d,e", [(4, 2, 24, 12), (3, 3, 40, 10), (1, 1, 16, 16), (4, 1, 64, 32), (2, 1, 130, 70), (8, 2, 128, 128), (40, 8, 128, 64), (2, 2, 8, 200)])
def test_delta_rule_with_a_decay_a_key_channel(H, G, d, e):
    """Unit vectors, step sizes, decays of every head and channel and the recurrence against the plain functions: two sequences
    side by side in portions of 1 to 40 tokens (one size also with a portion of 300 tokens of many heads), in state slots that
    held other contents, a padding sequence beside them, a step that keeps nothing."""
    from mini_rsglang_b200 import kernels

    gen = torch.Generator().manual_seed(d + e)
    lengths, cuts = ([97, 61], [[40, 1, 2, 1, 1, 33, 19], [1, 1, 3, 56]]) if H < 40 else ([307, 2], [[300, 7], [1, 1]])
    channels = 2 * G * d + H * e
    data = []
    for n in lengths:
        qkv, b, z = torch.randn(n, channels, generator=gen), torch.randn(n, H, generator=gen) * 2, torch.randn(n, H * d, generator=gen) * 2
        data.append((qkv, b, z))
    a_log, dt_bias = torch.randn(H, generator=gen) - 2, torch.randn(H * d, generator=gen) - 1
    a_log[0] = 3.0                                           # a head that forgets almost everything
    want = []
    for qkv, b, z in data:
        n = qkv.shape[0]
        q = P.unit(qkv[:, :G * d].double().view(n, G, d)) * d ** -0.5
        k = P.unit(qkv[:, G * d:2 * G * d].double().view(n, G, d))
        v = qkv[:, 2 * G * d:].double().view(n, H, e)
        x = z.double() + dt_bias.double()
        decay = torch.exp(-torch.exp(a_log.double())[None, :, None] * torch.nn.functional.softplus(x).view(n, H, d))
        want.append(torch.stack([P.channel_delta_recurrence(q[:, h // (H // G)], k[:, h // (H // G)], v[:, h], torch.sigmoid(b[:, h].double()),
                                                            decay[:, h])[0] for h in range(H)], dim=1).reshape(n, H * e))
    state = torch.full((3, 5 + H * d * e), 11.0, device=DEV)
    S = state[:, 5:].view(3, H, d, e)
    for index, batch in enumerate(steps_of(lengths, cuts)):
        qkv, b, z = (torch.cat([data[s][i][first:first + n] for s, first, n in batch]).to(DEV).contiguous() for i in range(3))
        positions, q_start, slots = step_facts(batch, [2, 0])
        wide = torch.cat([z, torch.randn(z.shape[0], 4, device=DEV)], dim=1).contiguous()
        fades = wide[:, :H * d]
        coef, out = torch.empty(z.shape[0], H, device=DEV), torch.zeros(z.shape[0], H * e, device=DEV)
        kernels.delta_prepare(qkv, b, 0, 0, a_log.to(DEV), dt_bias.to(DEV), coef, G, d, H, e, 1e-6, d ** -0.5, channels=fades)
        for write in ((False, True) if index == 1 else (True,)):
            before = state.clone()
            kernels.delta_scan(qkv, coef, S, positions, q_start, slots, out, H, G, d, e, write_state=write, channels=fades)
            assert write or torch.equal(before, state), "a step that keeps nothing wrote the state"
        at = 0
        for s, first, n in batch:
            w = want[s][first:first + n]
            assert (out[at:at + n].double().cpu() - w).abs().max() < 2e-4 * max(1.0, want[s].abs().max().item()), (s, first)
            at += n
    assert (state[1] == 11.0).all() and (state[:, :5] == 11.0).all()


def test_a_channel_decay_acts_on_its_own_row():
    """Two keys along two channels, one of which forgets: hundreds of decoded tokens later the value under the lasting channel is
    read back whole and the other one's is gone."""
    from mini_rsglang_b200 import kernels

    d, e, n = 8, 4, 300
    values = torch.randn(2, e)
    S = torch.full((2, 1, d, e), 5.0, device=DEV)
    outs = []
    for t in range(n):
        qkv = torch.zeros(1, 2 * d + e)
        if t < 2:
            qkv[0, d + 1 + 4 * t] = 1.0                      # keys along the channels 1 and 5
            qkv[0, 2 * d:] = values[t]
        if t >= n - 2:
            qkv[0, 1 + 4 * (t - (n - 2))] = 1.0              # queries along the same channels
        z = torch.full((1, d), -40.0)
        z[0, 5] = 0.0 if t >= 2 else -40.0                   # channel 5 halves, token by token
        b = torch.full((1, 1), 40.0 if t < 2 else -40.0)
        qkv, z, b = qkv.to(DEV), z.to(DEV), b.to(DEV)
        coef, out = torch.empty(1, 1, device=DEV), torch.zeros(1, e, device=DEV)
        kernels.delta_prepare(qkv, b, 0, 0, torch.zeros(1, device=DEV), torch.zeros(d, device=DEV), coef, 1, d, 1, e, 1e-6, 1.0, channels=z)
        kernels.delta_scan(qkv, coef, S, torch.tensor([t], dtype=torch.int32, device=DEV), torch.tensor([0, 1], dtype=torch.int32, device=DEV),
                           torch.tensor([1], dtype=torch.int32, device=DEV), out, 1, 1, d, e, channels=z)
        outs.append(out.cpu())
    assert (outs[n - 2][0] - values[0]).abs().max() < 1e-5 * values.abs().max() + 2e-6
    assert outs[n - 1].abs().max() < 1e-30
    assert (S[0] == 5.0).all()


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


@pytest.mark.parametrize("gated", [False, True])
def test_a_sum_of_mixers_is_the_mixers_each_alone(gated):
    """Terms and sum, with one projection for both mixers and (an attention whose gates are columns of its own) without."""
    from mini_rsglang_b200.cache.storage import CacheEntry
    from mini_rsglang_b200.parts.base import MIXERS, PartSpec, Runtime
    from mini_rsglang_b200.weights import random_weights

    width, n, page = 24, 21, 4
    attention = PartSpec("biased_window_attention", {"width": width, "num_heads": 2, "num_kv_heads": 1, "head_dim": 10, "value_dim": 6,
                                                     "position": PartSpec("rope", {"head_dim": 10, "theta": 100.0}),
                                                     "output_gate": "elements" if gated else False})
    memory = PartSpec("matrix_memory", {"width": width, "heads": 3, "head_dim": 6, "value_dim": 10, "gate_cap": 5.0, "eps": 1e-5})
    both_of = MIXERS.build(PartSpec("mixer_sum", {"width": width, "branches": [("x", attention, 0.7), ("y", memory, -2.0)]}), "m")
    alone = [MIXERS.build(attention, "m.x"), MIXERS.build(memory, "m.y")]
    tensors = random_weights(both_of.weight_specs(), 3, torch.float32, DEV)
    tensors = {name: t * 10.0 for name, t in tensors.items()}
    for part in (both_of, *alone):
        part.bind(tensors, Runtime(torch.device(DEV), torch.float32, page))
    assert (both_of.fused is None) == gated

    def cache():
        return CacheEntry(group=0, k=torch.zeros(6, 1, page, 10, device=DEV), v=torch.zeros(6, 1, page, 6, device=DEV),
                          state=torch.full((2, *both_of.state_need().shape), 3.0, device=DEV))

    torch.manual_seed(1)
    h = torch.randn(n, width, device=DEV)
    table = torch.randperm(6).to(torch.int32)
    caches = [cache() for _ in range(3)]
    for at, m in ((0, 15), (15, 1), (16, 5)):
        places = torch.arange(at, at + m)
        ctx = one_sequence(at, m, table, table.long()[places // page] * page + places % page)
        x = h[at:at + m].contiguous()
        want = 0.7 * alone[0].forward(x, ctx, caches[0]).double() - 2.0 * alone[1].forward(x, ctx, caches[0]).double()
        got = both_of.forward(x, ctx, caches[1])
        terms = both_of.forward(x, ctx, caches[2], as_terms=True).terms
        scale = want.abs().max()
        assert scale > 1e-3 and (got.double() - want).abs().max() < 1e-5 * scale
        assert (sum(f * t.double() for t, f in terms) - want).abs().max() < 1e-5 * scale


def test_the_stream_after_every_layer(folders, tmp_path_factory):
    """`bin/trace_run --observe`: the float32 residual stream after the embedding and after every layer run against the plain
    implementation, in a prompt's portion and in decoded tokens."""
    import numpy as np

    config, weights = load_plain(folders["X"])
    tokens = T.requests_for(config["vocab"], [19], seed=77)["r0"]
    layers = []
    P.forward(config, weights, tokens, layers_out=layers)
    out = str(tmp_path_factory.mktemp("observed"))
    run = T.TraceRun(folders["X"], "float32", out, 64, extra=("--page-size", "4", "--observe", "a"))
    for step, (at, m) in enumerate(((0, 16), (16, 1), (17, 2))):
        run.step({"step": step, "entries": [{"id": "a", "tokens": tokens[at:at + m], "want": []}], "end": []}, config["vocab"])
        for i, stream in enumerate(layers):
            got = np.fromfile(os.path.join(out, "observe", f"{step}.layer{i}-output.f32"), dtype="<f4").reshape(m, config["width"])
            want = stream[at:at + m]
            assert (torch.from_numpy(got).double() - want).abs().max() < 2e-5 * max(1.0, want.abs().max().item()), (step, i)
    assert run.close() == 0


@pytest.mark.parametrize("H,G,d,e,page", [(6, 2, 20, 12, 4), (4, 2, 64, 64, 16), (8, 1, 32, 48, 16), (8, 1, 64, 128, 16), (2, 1, 128, 128, 16)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_attention_reads_far_keys_and_page_borders(tmp_path_factory, H, G, d, e, page, dtype):
    """The attention of a "parallel" layer as the engine builds it, on one sequence in portions and decoded tokens: each of some
    places (the first tokens, both sides of page borders, far back, the last one) is the only key that answers the queries, whose
    output is then that place's value."""
    from mini_rsglang_b200 import kernels
    from mini_rsglang_b200.cache.storage import CacheEntry
    from mini_rsglang_b200.parts.base import MIXERS, PartSpec, Runtime

    torch_dtype = getattr(torch, dtype)
    width, n = 16, 333
    part = MIXERS.build(PartSpec("biased_window_attention", {
        "width": width, "num_heads": H, "num_kv_heads": G, "head_dim": d, "value_dim": e, "scale": 0.5,
        "position": PartSpec("banded_rope", {"head_dim": d, "theta": 300.0, "rotary_dim": d // 4 * 2, "factor": 4.0, "low": 1.0, "high": 4.0,
                                             "original": 64})}), "a")
    eye = torch.eye(H * e)[:min(width, H * e)]
    o_proj = torch.zeros(width, H * e)
    o_proj[:eye.shape[0]] = eye
    tensors = {"a.q_proj.weight": torch.zeros(H * d, width), "a.k_proj.weight": torch.zeros(G * d, width), "a.v_proj.weight": torch.zeros(G * e, width),
               "a.o_proj.weight": o_proj}
    part.bind({k: t.to(torch_dtype).to(DEV) for k, t in tensors.items()}, Runtime(torch.device(DEV), torch_dtype, page))
    pages = -(-n // page)
    gen = torch.Generator().manual_seed(d)
    table = torch.randperm(pages + 3, generator=gen)[:pages].to(torch.int32)
    values = torch.randn(n, G, e, generator=gen).bfloat16().float()
    for place in (0, 1, page - 1, page, 5 * page - 1, 5 * page, 200, 299):
        proj = torch.zeros(n, (H + G) * d + G * e)
        proj[:, d - 1:H * d:d] = 12.0                        # the last element of a head does not turn
        proj[place, H * d + d - 1:(H + G) * d:d] = 12.0
        proj[:, (H + G) * d:] = values.reshape(n, G * e)
        cache = CacheEntry(group=0, k=torch.full((pages + 3, G, page, d), 7.0, dtype=torch_dtype, device=DEV),
                           v=torch.full((pages + 3, G, page, e), -9.0, dtype=torch_dtype, device=DEV))
        cuts = [300, 2, 21] + [1] * 10
        at = 0
        for m in cuts:
            positions = torch.arange(at, at + m, dtype=torch.int32)
            slots = table.long()[positions.long() // page] * page + positions % page
            ctx = one_sequence(at, m, table, slots)
            out = part.forward_projected(proj[at:at + m].to(DEV).contiguous(), 0, ctx, cache).cpu()
            kernels.check_device_errors()
            first = max(place - at, 0)
            want = torch.cat([values[place, h // (H // G)] for h in range(H)])[:eye.shape[0]]
            got = out[first:, :eye.shape[0]]
            assert got.numel() == 0 or (got - want).abs().max() < 0.02, (place, at, m)
            at += m


# ----------------------------------------------------------------------------------------------------------------
# the engine's own entry point and scheduler
# ----------------------------------------------------------------------------------------------------------------
def check_greedy(config, weights, prompt, generated, dtype):
    """Every generated token is the plain implementation's arg-max behind what came before it, or within rounding of it."""
    logits = P.forward(config, weights, list(prompt) + list(generated))
    for i, token in enumerate(generated):
        row = logits[len(prompt) - 1 + i]
        gap = (row.max() - row[token]).item()
        limit = 2e-5 * max(1.0, row.abs().max().item()) if dtype == "float32" else 0.02 * row.abs().max().item()
        assert gap <= limit, f"{dtype}: engine chose {token}, plain {int(row.argmax())}, gap {gap}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["X", "Y"])
def test_greedy_generation_through_the_engine(folders, name, dtype):
    """Prompts of unequal lengths, more requests than run at a time (state slots are used again), prompt portions under a small
    token budget beside decoded tokens, 60 generated tokens each."""
    from mini_rsglang_b200 import RuntimeConfig, SamplingParams
    from mini_rsglang_b200.engine import EngineHandle

    config, weights = load_plain(folders[name])
    prompts = [T.requests_for(config["vocab"], [n], seed=500 + n)["r0"] for n in (3, 50, 1, 77, 20, 31)]
    engine = EngineHandle.load(folders[name], 0, config=RuntimeConfig(max_seq_len=160, prefill_budget=24, max_running=3, page_size=SHAPES[name][1]),
                               dtype=dtype, num_pages=120 if name == "X" else 40)
    results = engine.generate_many(prompts, SamplingParams(max_tokens=60, ignore_eos=True))
    engine.shutdown()
    for prompt, result in zip(prompts, results):
        assert len(result.token_ids) == 60
        check_greedy(config, weights, prompt, result.token_ids, dtype)


def test_one_request_at_a_time(folders):
    """An engine with a single state slot."""
    from mini_rsglang_b200 import RuntimeConfig, SamplingParams
    from mini_rsglang_b200.engine import EngineHandle

    config, weights = load_plain(folders["X"])
    engine = EngineHandle.load(folders["X"], 0, config=RuntimeConfig(max_seq_len=64, prefill_budget=64, max_running=1, page_size=4),
                               dtype="float32", num_pages=16)
    prompts = [[5, 9, 2, 200, 17], [8, 8]]
    for prompt, result in zip(prompts, engine.generate_many(prompts, SamplingParams(max_tokens=8, ignore_eos=True))):
        check_greedy(config, weights, prompt, result.token_ids, "float32")
    engine.shutdown()


def test_command_line_generates_the_plain_tokens(folders):
    import subprocess
    import sys

    prompt = [3, 1, 4, 1, 5, 9, 2, 6]
    cmd = [sys.executable, os.path.join(T.ROOT, "bin", "mini-rsglang"), "--model", folders["X"], "--dtype", "float32", "--page-size", "4",
           "--max-seq-len", "128", "--num-pages", "40", "generate", "--token-ids", ",".join(map(str, prompt)), "--max-tokens", "12",
           "--ignore-eos", "--json"]
    proc = subprocess.run(cmd, capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr
    events = [json.loads(line) for line in proc.stdout.splitlines() if line.startswith("{")]
    tokens = [e["Token"]["token_id"] for e in events if "Token" in e]
    assert events[-1]["Finished"]["completion_tokens"] == 12 == len(tokens)
    check_greedy(*load_plain(folders["X"]), prompt, tokens, "float32")
