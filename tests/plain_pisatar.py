"""A plain, slow implementation of the Pisatar design: one function per mechanism, written from the design's
equations with torch on the CPU (float64 unless told otherwise).  It is the oracle of the tests and shares no
code with the engine: it reads the configuration as a plain dict and the weights as a dict of tensors under
their checkpoint names, runs one whole sequence at a time and keeps nothing between calls.

Notation: T tokens, W width, H heads, G key/value (or query/key) heads, d the query/key size of a head, e the
value size of a head, C the taps of a convolution."""
from __future__ import annotations

import math

import torch


def over_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def shifted_norm(x, w, eps):
    """An RMS norm whose weight is stored as its distance from one."""
    return over_rms(x, eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


def plain_frequencies(rot):
    return [rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)]


def stretched_frequencies(rot):
    """Pairs with short wavelengths keep their frequency, long ones are slowed down by `factor`, and between the two bounds
    the frequency runs linearly from one to the other in (original length / wavelength)."""
    s = rot.get("scaling")
    out = []
    for f in plain_frequencies(rot):
        if s:
            wavelength = 2.0 * math.pi / f
            if wavelength > s["original"] / s["low"]:
                f = f / s["factor"]
            elif not wavelength < s["original"] / s["high"]:
                t = (s["original"] / wavelength - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - t) * f / s["factor"] + t * f
        out.append(f)
    return out


def rotate(x, frequencies, positions=None):
    """x [T, heads, d]: element i turns with element i + n (n frequencies), by position * frequency; the rest passes."""
    T, n = x.shape[0], len(frequencies)
    if n == 0:
        return x
    p = torch.arange(T) if positions is None else torch.as_tensor(positions)
    angle = p.to(torch.float64)[:, None] * torch.tensor(frequencies, dtype=torch.float64)[None, :]
    c, s = torch.cos(angle).to(x.dtype)[:, None, :], torch.sin(angle).to(x.dtype)[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], dim=-1)


def retention_recurrence(q, k, v, decay, state=None):
    """One head: q, k [T, d], v [T, e].  S <- decay S + k v^T; o = S^T q.  Returns (o, the last S)."""
    T, d = q.shape
    S = torch.zeros(d, v.shape[1], dtype=q.dtype) if state is None else state.clone()
    o = torch.empty(T, v.shape[1], dtype=q.dtype)
    for t in range(T):
        S = decay * S + torch.outer(k[t], v[t])
        o[t] = S.T @ q[t]
    return o, S


def retention(h, w, p, c, eps):
    T, H, d, e = h.shape[0], c["heads"], c["dim"], c["vdim"]
    f = plain_frequencies(c["rot"])
    q = rotate((h @ w[p + "q"].T).view(T, H, d), f)
    k = rotate((h @ w[p + "k"].T).view(T, H, d), f) * d ** -0.5
    v = (h @ w[p + "v"].T).view(T, H, e)
    o = torch.stack([retention_recurrence(q[:, i], k[:, i], v[:, i], c["decay"][i])[0] for i in range(H)], dim=1)
    return (over_rms(o, eps).reshape(T, H * e) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def causal_conv_silu(x, taps):
    """x [T, channels], taps [channels, C]: y_t = sum_c taps[:, c] x_(t - (C - 1) + c), zeros before the start; then silu."""
    T, channels = x.shape
    C = taps.shape[1]
    padded = torch.cat([torch.zeros(C - 1, channels, dtype=x.dtype), x], dim=0)
    y = torch.zeros_like(x)
    for c in range(C):
        y = y + padded[c:c + T] * taps[:, c]
    return silu(y)


def unit(x, eps=1e-6):
    return x / torch.sqrt(x.pow(2).sum(dim=-1, keepdim=True) + eps)


def channel_delta_recurrence(q, k, v, beta, decay, state=None):
    """One head: q, k, decay [T, d], v [T, e], beta [T].  Row i of S forgets by decay[t, i]; u = beta (v - S^T k);
    S <- S + k u^T; o = S^T q.  Returns (o, the last S)."""
    T, d = q.shape
    S = torch.zeros(d, v.shape[1], dtype=q.dtype) if state is None else state.clone()
    o = torch.empty(T, v.shape[1], dtype=q.dtype)
    for t in range(T):
        S = decay[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        o[t] = S.T @ q[t]
    return o, S


def channel_decay(h, w, p, H, d):
    """[T, H, d]: exp(-exp(A_log of the head) * softplus(two thin products + dt_bias))."""
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    softplus = torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30))))
    return torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * softplus.view(-1, H, d))


def channel_delta(h, w, p, c, eps):
    T = h.shape[0]
    H, G, d, e = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = unit(causal_conv_silu(h @ w[p + "q"].T, w[p + "q.conv"]).view(T, G, d)) * d ** -0.5
    k = unit(causal_conv_silu(h @ w[p + "k"].T, w[p + "k.conv"]).view(T, G, d))
    v = causal_conv_silu(h @ w[p + "v"].T, w[p + "v.conv"]).view(T, H, e)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    decay = channel_decay(h, w, p, H, d)
    o = torch.stack([channel_delta_recurrence(q[:, i // (H // G)], k[:, i // (H // G)], v[:, i], beta[:, i], decay[:, i])[0]
                     for i in range(H)], dim=1)
    o = (over_rms(o, eps) * w[p + "norm"]).reshape(T, H * e) * torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
    return o @ w[p + "o"].T


def grouped_attention(q, k, v, scale):
    """q [T, H, d], k [T, G, d], v [T, G, e]: causal softmax, head h over the keys of head h // (H / G); [T, H, e]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    seen = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    out = []
    for i in range(H):
        g = i // (H // G)
        s = torch.where(seen, q[:, i] @ k[:, g].T * scale, torch.tensor(-math.inf, dtype=q.dtype))
        out.append(torch.softmax(s, dim=-1) @ v[:, g])
    return torch.stack(out, dim=1)


def rotary_attention(h, w, p, c):
    T, H, G, d, e = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    f = stretched_frequencies(c["rot"])
    q = rotate((h @ w[p + "q"].T).view(T, H, d), f)
    k = rotate((h @ w[p + "k"].T).view(T, G, d), f)
    v = (h @ w[p + "v"].T).view(T, G, e)
    return grouped_attention(q, k, v, c["scale"]).reshape(T, H * e) @ w[p + "o"].T


def capped(z, cap):
    return cap * torch.tanh(z / cap)


def log_sigmoid(z):
    return -(torch.clamp(-z, min=0) + torch.log1p(torch.exp(-z.abs())))


def memory_recurrence(q, k, v, log_in, log_keep, state=None):
    """One head: q, k [T, d], v [T, e], log_in, log_keep [T].  m' = max(keep + m, in); S and n forget by exp(keep + m - m')
    and take exp(in - m') k v^T (k alone); o = S^T q / (max(|n . q|, exp(-m')) + 1e-6).  m starts at 0.
    Returns (o, (S, n, m))."""
    T, d = q.shape
    if state is None:
        S, n, m = torch.zeros(d, v.shape[1], dtype=q.dtype), torch.zeros(d, dtype=q.dtype), torch.zeros((), dtype=q.dtype)
    else:
        S, n, m = (x.clone() for x in state)
    o = torch.empty(T, v.shape[1], dtype=q.dtype)
    for t in range(T):
        top = torch.maximum(log_keep[t] + m, log_in[t])
        keep, take = torch.exp(log_keep[t] + m - top), torch.exp(log_in[t] - top)
        S = keep * S + take * torch.outer(k[t], v[t])
        n = keep * n + take * k[t]
        m = top
        o[t] = S.T @ q[t] / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + 1e-6)
    return o, (S, n, m)


def matrix_memory(h, w, p, c, eps):
    T, H, d, e, cap = h.shape[0], c["heads"], c["dim"], c["vdim"], c["gate_cap"]
    q = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, d)
    v = (h @ w[p + "v"].T).view(T, H, e)
    log_in = capped(h @ w[p + "i"].T + w[p + "i.b"], cap)
    log_keep = log_sigmoid(capped(h @ w[p + "f"].T + w[p + "f.b"], cap))
    o = torch.stack([memory_recurrence(q[:, i], k[:, i], v[:, i], log_in[:, i], log_keep[:, i])[0] for i in range(H)], dim=1)
    return (over_rms(o, eps).reshape(T, H * e) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(h, w, p, c, eps):
    return (c["left_scale"] * rotary_attention(h, w, p + "left.", c["left"])
            + c["right_scale"] * matrix_memory(h, w, p + "right.", c["right"], eps))


def gated_mlp(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


MIXERS = {"retention": retention, "channel_delta": channel_delta, "parallel": parallel}


def weights_index(config: dict, i: int) -> int:
    """The layer whose tensors layer i uses."""
    seen = set()
    while config["layers"][i].get("weights_of") is not None and i not in seen:
        seen.add(i)
        i = config["layers"][i]["weights_of"]
    return i


def forward(config: dict, w: dict, tokens, dtype=torch.float64, layers_out: list | None = None):
    """Logits [T, vocab] of one sequence from position 0.  `layers_out`: a list that gets the residual stream
    after every layer."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps = config["norm"]["eps"]
    x = shifted_norm(w["embed"][torch.as_tensor(tokens, dtype=torch.long)], w["embed.norm"], eps)
    for i, layer in enumerate(config["layers"]):
        p = f"l{weights_index(config, i)}."
        y = MIXERS[layer["type"]](shifted_norm(x, w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + gated_mlp(shifted_norm(x, w[p + "norm2"], eps), w, p + "mlp.")
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return shifted_norm(x, w["final.norm"], eps) @ w["head"].T
