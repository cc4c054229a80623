"""A plain, slow implementation of the Bilipel design: one function per mechanism, written from the design's
equations with torch on the CPU (float64 unless told otherwise).  It is the oracle of the tests and shares no
code with the engine: it reads the configuration as a plain dict and the weights as a dict of tensors under
their checkpoint names, runs one whole sequence at a time and keeps nothing between calls.

Notation: T tokens, W width, H heads, G key/value heads, d the query/key size of a head, r its rotated part where that
stands apart, e the value size of a head, R the size of a latent, n the frequencies of a rotation."""
from __future__ import annotations

import math

import torch


def layer_norm(x, w, b, eps):
    """(x - mean) / sqrt(variance + eps) * w + b over the last dimension; the variance is the mean squared deviation."""
    y = x - x.mean(dim=-1, keepdim=True)
    return y / torch.sqrt(y.pow(2).mean(dim=-1, keepdim=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def plain_frequencies(base, dims):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def stretched_frequencies(base, dims, s):
    """(frequencies, factor on cosines and sines): pairs that turn often over the original length keep their frequency,
    those that hardly turn are slowed down by `factor`, a ramp over the pair's number in between."""
    def pair_of(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_of(s["fast"])), 0)
    hi = min(math.ceil(pair_of(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain_frequencies(base, dims)):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def angles(positions, frequencies, dtype, magnitude=1.0):
    """Cosines and sines [T, 1, n] of position * frequency."""
    a = torch.as_tensor(positions).to(torch.float64)[:, None] * torch.tensor(frequencies, dtype=torch.float64)[None, :]
    return (torch.cos(a) * magnitude).to(dtype)[:, None, :], (torch.sin(a) * magnitude).to(dtype)[:, None, :]


def rotate_halves(x, positions, frequencies, magnitude=1.0):
    """x [T, heads, d]: element i turns with element i + n, the elements from 2 n on pass."""
    n = len(frequencies)
    c, s = angles(positions, frequencies, x.dtype, magnitude)
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], dim=-1)


def rotate_neighbours(x, positions, frequencies):
    """x [T, heads, d]: element 2 i turns with element 2 i + 1, the elements from 2 n on pass."""
    n = len(frequencies)
    c, s = angles(positions, frequencies, x.dtype)
    u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
    out = x.clone()
    out[..., 0:2 * n:2], out[..., 1:2 * n:2] = u * c - v * s, v * c + u * s
    return out


def seen_in_window(T, window=0):
    """[T, T] bool: key j is seen by query i when j <= i and, with a window, i - j < window."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) & (back < window) if window else back >= 0


def softmax_with_sink(scores, seen, sink):
    """Weights of the keys; the denominator also has exp(sink), which has no key."""
    s = torch.where(seen, scores, torch.tensor(-math.inf, dtype=scores.dtype))
    top = torch.maximum(s.max(dim=-1, keepdim=True).values, sink)
    weights = torch.exp(s - top)
    return weights / (weights.sum(dim=-1, keepdim=True) + torch.exp(sink - top))


def attention_core(q, k, v, scale, sink):
    """q [T, H, d], k [T, G, d], v [T, G, e]: causal, head h over the keys of head h // (H / G); [T, H, e]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    seen = seen_in_window(T)
    out = []
    for h in range(H):
        g = h // (H // G)
        out.append(softmax_with_sink(q[:, h] @ k[:, g].T * scale, seen, sink[h]) @ v[:, g])
    return torch.stack(out, dim=1)


def attention(h, w, p, c, eps):
    T, H, G, d, e = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = rms_norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).view(T, H, d)          # one norm over all heads' rows
    k = rms_norm(h @ w[p + "k"].T, w[p + "k.norm"], eps).view(T, G, d)
    v = (h @ w[p + "v"].T).view(T, G, e)
    rot = c["rot"]
    if rot.get("scaling"):
        f, m = stretched_frequencies(rot["base"], rot["dims"], rot["scaling"])
    else:
        f, m = plain_frequencies(rot["base"], rot["dims"]), 1.0
    q, k = (rotate_halves(x, range(T), f, m) for x in (q, k))
    return attention_core(q, k, v, c["scale"], w[p + "sink"]).reshape(T, H * e) @ w[p + "o"].T


def latent_core(q_plain, q_rot, c, k_rot, w_uk, w_uv, scale, sink, window):
    """q_plain [T, H, d], q_rot [T, H, r], latent c [T, R], k_rot [T, r]: every head's keys and values made from the latent;
    [T, H, e]."""
    T, H, d = q_plain.shape
    e = w_uv.shape[0] // H
    k = (c @ w_uk.T).view(T, H, d)
    v = (c @ w_uv.T).view(T, H, e)
    seen = seen_in_window(T, window)
    out = []
    for h in range(H):
        scores = (q_plain[:, h] @ k[:, h].T + q_rot[:, h] @ k_rot.T) * scale
        out.append(softmax_with_sink(scores, seen, sink[h]) @ v[:, h])
    return torch.stack(out, dim=1)


def latent_attention(h, w, p, c, eps):
    T, H, d, r, R = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["kv_rank"]
    q = (h @ w[p + "q"].T).view(T, H, d + r)
    low = h @ w[p + "dkv"].T
    latent = rms_norm(low[:, :R], w[p + "dkv.norm"], eps)
    f = plain_frequencies(c["rot"]["base"], c["rot"]["dims"])
    q_rot = rotate_neighbours(q[..., d:], range(T), f)
    k_rot = rotate_neighbours(low[:, None, R:], range(T), f)[:, 0]
    out = latent_core(q[..., :d], q_rot, latent, k_rot, w[p + "uk"], w[p + "uv"], c["scale"], w[p + "sink"], c["mask"]["size"])
    return out.reshape(T, -1) @ w[p + "o"].T


def gla_recurrence(q, k, v, alpha, state=None):
    """q, k, alpha [T, H, d], v [T, H, e]: row i of S forgets by alpha[t, i], then S <- S + k v^T; o = S^T q.
    Returns (o [T, H, e], the last S [H, d, e])."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    o = torch.empty(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(dim=1)
    return o, S


def log_sigmoid(z):
    return -(torch.clamp(-z, min=0) + torch.log1p(torch.exp(-z.abs())))


def gla_decay(h, w, p, c):
    """[T, H, d]: the sigmoid of two thin products and a bias, to the power 1 / tau."""
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    return torch.exp(log_sigmoid(z) / c["tau"]).view(h.shape[0], c["heads"], c["dim"])


def gla(h, w, p, c, eps):
    T, H, d, e = h.shape[0], c["heads"], c["dim"], c["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, d)
    v = (h @ w[p + "v"].T).view(T, H, e)
    o, _ = gla_recurrence(q, k, v, gla_decay(h, w, p, c))
    o = rms_norm(o, w[p + "norm"], eps).reshape(T, H * e)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def gated_unit(h, w, p, act):
    return (act(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def choose_experts(z, top):
    """Router logits z [T, experts] -> (chosen [T, top], weights [T, top]): the softmax over the chosen logits only."""
    best = torch.topk(z, top, dim=-1)
    return best.indices, torch.softmax(best.values, dim=-1)


def experts(h, w, p, c):
    chosen, weights = choose_experts(h @ w[p + "router"].T + w[p + "router.b"], c["router"]["top"])
    out = torch.zeros_like(h)
    for number in range(c["router"]["experts"]):
        rows, place = (chosen == number).nonzero(as_tuple=True)
        if len(rows):
            out[rows] += weights[rows, place, None] * gated_unit(h[rows], w, f"{p}e{number}.", silu)
    return out


def feed_forward(h, w, p, c):
    return gated_unit(h, w, p, gelu_tanh) if c["kind"] == "dense" else experts(h, w, p, c)


MIXERS = {"attention": attention, "latent_attention": latent_attention, "gla": gla}


def run_order(c):
    """[(layer, number of the pass where one begins right before this run, else None)]."""
    n, loop = len(c["layers"]), c.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], n)]


def one_layer(x, w, i, c):
    layer, eps, m = c["layers"][i], c["norm"]["eps"], c.get("residual_mult", 1.0)
    p = f"l{i}."
    h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
    x = x + m * MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps)
    if layer.get("mlp") is not None:
        h = layer_norm(x, w[p + "norm2"], w[p + "norm2.b"], eps)
        x = x + m * feed_forward(h, w, p + "mlp.", layer["mlp"])
    return x


def enter_pass(x, origin, w, t):
    """What stands right before pass t of the loop."""
    return (x + origin if t else x) + w["loop.step"][t]


def logits_of_sequence(c, w, tokens, keep_layers=None):
    """Logits [T, vocab] of one whole sequence; `keep_layers` (a list) receives the stream after every layer run."""
    x = w["embed"][torch.as_tensor(tokens)]
    origin = x
    for i, t in run_order(c):
        if t is not None:
            x = enter_pass(x, origin, w, t)
        x = one_layer(x, w, i, c)
        if keep_layers is not None:
            keep_layers.append(x)
    return layer_norm(x, w["final.norm"], w["final.norm.b"], c["norm"]["eps"]) @ w["head"].T


def load(folder, dtype=torch.float64):
    """(configuration, weights) of a checkpoint folder, read without the engine."""
    import json
    import os

    from safetensors.torch import load_file

    with open(os.path.join(folder, "config.json")) as f:
        c = json.load(f)
    return c, {name: t.to(dtype) for name, t in load_file(os.path.join(folder, "model.safetensors")).items()}
