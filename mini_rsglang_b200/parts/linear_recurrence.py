"""Mixers whose state is a matrix a head, S [d, e], and linear in what they add to it.

"retention": linear attention with a constant decay a head, without softmax or denominator.  With h the mixer's input, H heads
of d query/key and e value elements:

  q = R(W_q h), k = R(W_k h) d^(-1/2)  [H, d]   (R: a registered position encoding, on part of a head or all of it);  v = W_v h  [H, e]
  S <- decay_head S + k v^T;  o = S^T q
  out = W_o (o / rms(o) * silu(W_g h))                                    rms over a head's e elements, no weight

"matrix_memory": an exponentially gated memory with a normaliser n [d] and a running maximum m, all three starting at zero:

  q = W_q h d^(-1/2), k = W_k h  [H, d];  v = W_v h  [H, e]
  i = cap tanh((W_i h + b_i) / cap), f = logsigmoid(cap tanh((W_f h + b_f) / cap))                 one each a head
  m' = max(f + m, i);  S <- exp(f + m - m') S + exp(i - m') k v^T;  n likewise with k alone;  m <- m'
  o = S^T q / (max(|n . q|, exp(-m)) + floor_eps)
  out = W_o (o / rms(o) * w_norm * sigmoid(W_g h))                        rms over a head, w_norm of all heads' size

"gated_linear_attention": one decay a key channel and token, which acts on the rows of S, from two thin products:

  q = W_q h d^(-1/2), k = W_k h  [H, d];  v = W_v h  [H, e];  a = sigmoid(W_a2 (W_a1 h) + b)^(1 / tau)  [H, d]
  S <- diag(a) S + k v^T;  o = S^T q
  out = W_o (o / rms(o) * w_norm * silu(W_g h))                           rms over a head, w_norm of a head's size

A request's state lives in its state slot as one float32 vector (S of every head, then n, then m) and counts as zero where a
sequence starts at position 0.  One projection gives everything that is read of h as float32 sums; rotation, gates, maxima,
recurrence and head norm are float32 (`kernels.linear_scan`; the factors d^(-1/2) are applied to the read-out, which is linear
in them).  Every size and constant is a parameter."""
from __future__ import annotations

import torch

from .. import kernels
from ..errors import InvalidRequest
from ..weights.spec import WeightSpec
from .base import MIXERS, POSITION_ENCODINGS, Mixer, PartSpec, StateNeed
from .linear import linear


class LinearRecurrence(Mixer):
    """What the two mixers share: the fused projection q | k | v | gate | ..., padded to rows of a multiple of 8."""

    replayable = True      # the step's facts are read from device tensors only
    PROJECTED: tuple[str, ...] = ()

    def __init__(self, prefix: str, width: int, heads: int, head_dim: int, value_dim: int, eps: float, names: dict | None):
        super().__init__(prefix)
        self.width, self.heads, self.d, self.e, self.eps = int(width), int(heads), int(head_dim), int(value_dim), float(eps)
        if min(self.width, self.heads, self.d, self.e) <= 0 or self.d > kernels.LINEAR_SCAN_MAX_DIM:
            raise InvalidRequest(f"{prefix}: sizes must be positive, query/key heads at most {kernels.LINEAR_SCAN_MAX_DIM} elements")
        self.leaf = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "gate": "g_proj.weight", "o": "o_proj.weight"}
        self.leaf.update(names or {})
        self.fused = self.w_o = None

    def weight_specs(self):
        n, qk, inner = self.leaf, self.heads * self.d, self.heads * self.e
        return [WeightSpec(self.name(n["q"]), (qk, self.width)), WeightSpec(self.name(n["k"]), (qk, self.width)),
                WeightSpec(self.name(n["v"]), (inner, self.width)), WeightSpec(self.name(n["gate"]), (inner, self.width)),
                WeightSpec(self.name(n["o"]), (self.width, inner))]

    def bind(self, tensors, runtime):
        super().bind(tensors, runtime)
        rows = [tensors[self.name(self.leaf[key])] for key in self.PROJECTED]
        padding = -sum(t.shape[0] for t in rows) % 8              # rows of the projection's sums on 16-byte boundaries
        rows += [rows[0].new_zeros((padding, self.width))] if padding else []
        self.fused = torch.cat(rows, dim=0).contiguous()
        self.w_o = tensors[self.name(self.leaf["o"])].contiguous()

    def projection(self):
        return self.fused

    def forward(self, h, ctx, cache, write_cache=True):
        return self.forward_projected(linear(h, self.fused, out_dtype=torch.float32), 0, ctx, cache, write_cache)

    def matrix_state(self, cache):
        """S of every head and slot: [slots, heads, d, e]."""
        return cache.state[:, :self.heads * self.d * self.e].view(cache.state.shape[0], self.heads, self.d, self.e)


@MIXERS.register("retention")
class Retention(LinearRecurrence):
    PROJECTED = ("q", "k", "v", "gate")

    def __init__(self, prefix: str, width: int, heads: int, head_dim: int, value_dim: int, decay: list, eps: float,
                 position: PartSpec | None = None, names: dict | None = None):
        """`decay`: one constant a head; `position`: how query and key heads turn (None: not at all)."""
        super().__init__(prefix, width, heads, head_dim, value_dim, eps, names)
        self.decay_values = [float(x) for x in decay]
        if len(self.decay_values) != self.heads:
            raise InvalidRequest(f"{prefix}: {len(self.decay_values)} decays for {self.heads} heads")
        self.position = POSITION_ENCODINGS.build(position, prefix) if position is not None else None

    def state_need(self):
        return StateNeed((self.heads * self.d * self.e,), torch.float32)

    def bind(self, tensors, runtime):
        super().bind(tensors, runtime)
        self.decay = torch.tensor(self.decay_values, dtype=torch.float32, device=runtime.device)
        if self.position is not None:
            self.position.bind(tensors, runtime)
            rotation = self.position.rotation()
            if rotation is not None and (rotation.pairing != "split_half" or rotation.magnitude != 1.0 or rotation.rotary_dim > self.d):
                raise InvalidRequest(f"{self.prefix}: heads turn in split halves, with unscaled cosines and sines")

    def forward_projected(self, proj, offset, ctx, cache, write_cache=True):
        tokens, device = proj.shape[0], proj.device
        H, d, e = self.heads, self.d, self.e
        k_at, v_at = offset + H * d, offset + 2 * H * d
        rotation = self.position.rotation() if self.position is not None else None
        if rotation is not None and rotation.rotary_dim:
            kernels.rotate_heads_(proj, offset, 2 * H, d, self.position.rotations(ctx), rotation.rotary_dim)
        o = torch.empty((tokens, H * e), dtype=torch.float32, device=device)
        kernels.linear_scan(proj, offset, k_at, v_at, self.decay, None, self.matrix_state(cache), None, ctx.positions, ctx.q_start,
                            ctx.state_slots, o, None, H, d, e, write_state=write_cache)
        normed = torch.empty((tokens, H * e), dtype=self.runtime.dtype, device=device)
        kernels.head_norm_gate(o, proj[:, v_at + H * e:v_at + 2 * H * e], None, self.eps, normed, H, factor=d ** -0.5)
        return linear(normed, self.w_o, out_dtype=torch.float32)


@MIXERS.register("matrix_memory")
class MatrixMemory(LinearRecurrence):
    PROJECTED = ("q", "k", "v", "gate", "i", "f")

    def __init__(self, prefix: str, width: int, heads: int, head_dim: int, value_dim: int, gate_cap: float, eps: float,
                 floor_eps: float = 1e-6, names: dict | None = None):
        super().__init__(prefix, width, heads, head_dim, value_dim, eps, dict({"i": "i_proj.weight", "f": "f_proj.weight", "i_bias": "i_proj.bias",
                                                                               "f_bias": "f_proj.bias", "norm": "norm.weight"}, **(names or {})))
        self.gate_cap, self.floor_eps = float(gate_cap), float(floor_eps)
        if not self.gate_cap > 0:
            raise InvalidRequest(f"{prefix}: the gates' cap must be positive")

    def weight_specs(self):
        n = self.leaf
        return super().weight_specs() + [
            WeightSpec(self.name(n["norm"]), (self.heads * self.e,), "vector"),
            WeightSpec(self.name(n["i"]), (self.heads, self.width)), WeightSpec(self.name(n["i_bias"]), (self.heads,), "bias"),
            WeightSpec(self.name(n["f"]), (self.heads, self.width)), WeightSpec(self.name(n["f_bias"]), (self.heads,), "bias")]

    def state_need(self):
        return StateNeed((self.heads * (self.d * self.e + self.d + 1),), torch.float32)

    def bind(self, tensors, runtime):
        super().bind(tensors, runtime)
        n = self.leaf
        self.norm_w = tensors[self.name(n["norm"])].float().contiguous()
        self.i_bias, self.f_bias = (tensors[self.name(n[key])].float().contiguous() for key in ("i_bias", "f_bias"))

    def forward_projected(self, proj, offset, ctx, cache, write_cache=True):
        tokens, device = proj.shape[0], proj.device
        H, d, e = self.heads, self.d, self.e
        k_at, v_at, g_at = offset + H * d, offset + 2 * H * d, offset + 2 * H * d + H * e
        i_at = g_at + H * e
        matrix, slots = H * d * e, cache.state.shape[0]
        n_state = cache.state[:, matrix:matrix + H * d].view(slots, H, d)
        m_state = cache.state[:, matrix + H * d:]
        coef = torch.empty((tokens, 3 * H), dtype=torch.float32, device=device)
        kernels.memory_gates(proj, i_at, i_at + H, self.i_bias, self.f_bias, self.gate_cap, m_state, ctx.positions, ctx.q_start,
                             ctx.state_slots, coef, write_state=write_cache)
        o = torch.empty((tokens, H * e), dtype=torch.float32, device=device)
        c = torch.empty((tokens, H), dtype=torch.float32, device=device)
        kernels.linear_scan(proj, offset, k_at, v_at, None, coef, self.matrix_state(cache), n_state, ctx.positions, ctx.q_start,
                            ctx.state_slots, o, c, H, d, e, write_state=write_cache)
        normed = torch.empty((tokens, H * e), dtype=self.runtime.dtype, device=device)
        kernels.head_norm_gate(o, proj[:, g_at:i_at], self.norm_w, self.eps, normed, H, gate_kind="sigmoid", factor=d ** -0.5,
                               normaliser=(c, coef[:, 2 * H:], self.floor_eps))
        return linear(normed, self.w_o, out_dtype=torch.float32)


@MIXERS.register("gated_linear_attention")
class GatedLinearAttention(LinearRecurrence):
    PROJECTED = ("q", "k", "v", "gate", "a_down")

    def __init__(self, prefix: str, width: int, heads: int, head_dim: int, value_dim: int, tau: float, eps: float, decay_rank: int = -1,
                 names: dict | None = None):
        """`tau`: the root that is taken of the sigmoid; `decay_rank`: inner size of the two thin products (-1: as the checkpoint
        has it)."""
        super().__init__(prefix, width, heads, head_dim, value_dim, eps, dict({"a_down": "a_down.weight", "a_up": "a_up.weight",
                                                                               "a_bias": "a_up.bias", "norm": "norm.weight"}, **(names or {})))
        self.tau, self.rank = float(tau), int(decay_rank)
        if not self.tau > 0:
            raise InvalidRequest(f"{prefix}: tau must be positive")

    def weight_specs(self):
        n, qk = self.leaf, self.heads * self.d
        return super().weight_specs() + [
            WeightSpec(self.name(n["norm"]), (self.e,), "vector"), WeightSpec(self.name(n["a_down"]), (self.rank, self.width)),
            WeightSpec(self.name(n["a_up"]), (qk, self.rank)), WeightSpec(self.name(n["a_bias"]), (qk,), "bias")]

    def state_need(self):
        return StateNeed((self.heads * self.d * self.e,), torch.float32)

    def bind(self, tensors, runtime):
        super().bind(tensors, runtime)
        n = self.leaf
        self.norm_w = tensors[self.name(n["norm"])].float().contiguous()
        self.a_up = tensors[self.name(n["a_up"])].contiguous()
        self.a_bias = tensors[self.name(n["a_bias"])].float().contiguous()
        self.rank = self.a_up.shape[1]
        if tensors[self.name(n["a_down"])].shape[0] != self.rank or self.rank > kernels.CHANNEL_SCAN_MAX_RANK:
            raise InvalidRequest(f"{self.prefix}: the thin products' inner sizes differ, or are above {kernels.CHANNEL_SCAN_MAX_RANK}")

    def forward_projected(self, proj, offset, ctx, cache, write_cache=True):
        tokens, device = proj.shape[0], proj.device
        H, d, e = self.heads, self.d, self.e
        k_at, v_at = offset + H * d, offset + 2 * H * d
        g_at, low_at = v_at + H * e, v_at + 2 * H * e
        o = torch.empty((tokens, H * e), dtype=torch.float32, device=device)
        kernels.channel_scan(proj, offset, k_at, v_at, low_at, self.a_up, self.a_bias, self.tau, self.matrix_state(cache), ctx.positions,
                             ctx.seq_of_token, ctx.q_start, ctx.state_slots, o, H, d, e, write_state=write_cache)
        normed = torch.empty((tokens, H * e), dtype=self.runtime.dtype, device=device)
        kernels.head_norm_gate(o, proj[:, g_at:low_at], self.norm_w, self.eps, normed, H, factor=d ** -0.5)
        return linear(normed, self.w_o, out_dtype=torch.float32)
