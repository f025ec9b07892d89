"""Mixers that carry a state of fixed size from token to token, and the mixer that runs two
mixers side by side.

``gated_linear_recurrence``: two branches of ``width`` channels from one projection of the
input, ``y = act(W_y x + b_y)`` and ``u = conv(W_x x + b_x)`` (a causal convolution per channel);
u is cut into ``blocks`` equal parts and in part b ``r = sigmoid(A[b] u_b + a[b])``,
``i = sigmoid(I[b] u_b + c[b])``; with ``log a = -decay_scale * r * softplus(lam)`` the state is
``S <- a S + sqrt(1 - a^2) * i * u`` from ``S = 0`` (the first token is no special case) and the
result ``W_o (S * y)``.  (The recurrent block of De et al., "Griffin: Mixing Gated Linear
Recurrences with Local Attention for Efficient Language Models".)

``state_space``: one projection of the input gives ``z | x | B | C | dt``; x, B and C pass a
causal convolution per channel and SiLU; per head h (heads share B and C in ``groups``)
``dt = softplus(dt + dt_bias_h)``, ``S <- exp(-exp(A_log_h) dt) S + dt B x^T`` (S is state_size x
value_dim), ``y = S^T C + D_h x``; then ``y * silu(z)``, an RMS norm in ``norm_groups`` equal
parts times a weight, and W_o.  (The SSD layer of Dao and Gu, "Transformers are SSMs".)

Both keep, per request, the last ``taps - 1`` inputs of their convolution and the recurrent
state S in one float32 row of the slot-indexed state array, which starts at zero when a request
takes its slot.  Gates, decays, step sizes and S are float32 whatever the compute dtype; the
projections run in the compute dtype.

``delta_rule``: the generalized delta rule.  ``heads`` heads of ``dim`` channels; one projection
of the input gives ``r | k | v | g | a | w1`` (the last ``decay_rank`` rows are the first half of
the decay's two small matrices).  In float32, per head and key channel, the decay is
``w = exp(-decay_scale * sigmoid(W_w2 tanh(W_w1 x) + w0))`` and the removal rate ``a = sigmoid(W_a x
+ a_bias)``; with the unit key ``u = k / sqrt(sum(k^2) + key_eps)`` the state (``dim`` x ``dim`` per
head, float32) goes ``S <- diag(w) S - (a * u)(u^T S) + k v^T``, both middle terms reading the old
state, and the head's result is ``S^T r``, divided by its root mean square, times a weight over all
heads' channels, times ``sigmoid(g)``, then W_o.

``gated_delta_rule``: the delta rule with a decay in front (Yang et al., "Gated Delta Networks: Improving
Mamba2 with Delta Rule").  q and k (``kv_heads`` x ``dim``) and v (``heads`` x ``value_dim``) pass a
causal convolution per channel and SiLU; q and k become unit vectors per head, q times ``dim^(-1/2)``;
head h reads key head ``h // (heads / kv_heads)``.  With the decay ``g = exp(-exp(A_log_h) softplus(a +
dt_bias))`` (``decay`` "head": one per head, "channel": one per head and key channel) and ``beta =
sigmoid(b)`` the state goes ``S <- g S;  S <- S + k (beta (v - S^T k))^T`` and the head's result is ``S^T
q``, divided by its root mean square, times a weight shared by the heads, times a gate (``silu`` or
``sigmoid``), then W_o.  The decay's logits and the gate's come from the layer's input directly or
through a low-rank pair.  (State: S and a ring of the convolution's last inputs.)

``selective_scan``: one projection of the input gives ``x | z`` (``inner`` channels each); x passes a causal convolution
per channel with a bias and SiLU; a second product of x gives ``low | B | C`` (``rank``, ``state_size``, ``state_size``) and a
third, of low, the step sizes' logits, ``dt = softplus(W_dt low + bias)`` per channel; with ``A = -exp(A_log)`` the
state of channel c goes ``S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n`` and the result is ``W_o ((sum_n S[c, n] C_n +
D_c x_c) * silu(z_c))``.  (Gu and Dao, "Mamba: Linear-Time Sequence Modeling with Selective State Spaces".)

``gated_linear_attention``: ``S <- diag(alpha) S + k v^T`` per head (``dim`` x ``value_dim``, float32) with ``alpha =
sigmoid(W_up (W_low x) + bias)^(1 / tau)`` per key channel, read by ``S^T (dim^(-1/2) q)``; every head's result is
divided by its root mean square, times a weight shared by the heads, times ``silu(W_g x)``, then W_o.  (Yang et al.,
"Gated Linear Attention Transformers with Hardware-Efficient Training".)

``side_by_side``: two mixers read the same input; the result is ``scale * (rms_norm(left) * w_l
+ rms_norm(right) * w_r)`` over the model width, or, with ``join`` = "weighted_sum",
``left_scale * left + right_scale * right`` without norms.
"""
from __future__ import annotations

import math

import torch

from ..ops import kernels
from ..ops.linear import SMALL_STEP_TOKENS, linear, use_tensor_core_kernel
from .base import CacheNeeds, Mixer, StateSpec, product_of
from .registry import part_class, register_part

_ACTS = {"none": kernels.ACT_NONE, "silu": kernels.ACT_SILU, "gelu_tanh": kernels.ACT_GELU_TANH,
         "relu_squared": kernels.ACT_RELU_SQUARED, "tanh": kernels.ACT_TANH}


def activation_code(name: str) -> int:
    try:
        return _ACTS[name]
    except KeyError:
        raise ValueError(f"unknown activation {name!r}; known: {sorted(_ACTS)}") from None


def _pad_rows(weight: torch.Tensor, multiple: int = 8) -> torch.Tensor:
    rows = weight.shape[0]
    width = -(-rows // multiple) * multiple
    if width == rows:
        return weight
    return torch.cat([weight, weight.new_zeros((width - rows,) + tuple(weight.shape[1:]))]).contiguous()


def _pad_cols(weight: torch.Tensor, width: int = 0, multiple: int = 8) -> torch.Tensor:
    """Columns of zeros up to ``width``, or to a multiple."""
    cols = weight.shape[1]
    width = width or -(-cols // multiple) * multiple
    if width <= cols:
        return weight.contiguous()
    return torch.cat([weight, weight.new_zeros(weight.shape[0], width - cols)], dim=1).contiguous()


def _lowered_rows(sums: torch.Tensor, ws, dtype, num_rows: int) -> torch.Tensor:
    """float32 rows in the compute dtype (for a block that has offered no stream to add into)."""
    if dtype == torch.float32:
        return sums
    out = ws.get("side_by_side.out", (ws.max_tokens, sums.shape[1]), dtype)
    kernels.cast_f32_to_bf16(sums, out, num_rows * sums.shape[1])
    return out


@register_part("mixer", "gated_linear_recurrence")
class GatedLinearRecurrence(Mixer):
    takes_padded_steps = True

    def __init__(self, params, weights, dtype, device, position=None) -> None:
        super().__init__(params, weights, dtype, device)
        self.hidden_size = E = int(params["hidden_size"])
        self.width = W = int(params["width"])
        self.blocks = int(params["blocks"])
        self.taps = int(params["conv_taps"])
        self.decay_scale = float(params.get("decay_scale", 8.0))
        self.branch_act = activation_code(params.get("branch_activation", "gelu_tanh"))
        if W % self.blocks != 0:
            raise ValueError(f"width={W} is not a multiple of blocks={self.blocks}")
        if self.taps < 1:
            raise ValueError("conv_taps must be at least 1")
        part = W // self.blocks
        # y | x in one projection.
        self.w_in = self.expect("in.weight", (2 * W, E))
        self.b_in = self.expect("in.bias", (2 * W,))
        self.in_width = -(-2 * W // 8) * 8
        self.w_in, self.b_in = _pad_rows(self.w_in), _pad_rows(self.b_in)
        self.b_in_lowp = self.b_in.to(dtype) if dtype != torch.float32 else None
        self.conv_w = self.expect("conv.weight", (W, self.taps))
        self.conv_b = self.expect("conv.bias", (W,))
        # The gate matrices are stored [block, out, in]; the kernel reads them [block, in, out].
        self.gate_a = self.expect("gate_a.weight", (self.blocks, part, part))
        self.gate_i = self.expect("gate_i.weight", (self.blocks, part, part))
        self.gate_a_t = self.gate_a.transpose(1, 2).contiguous()
        self.gate_i_t = self.gate_i.transpose(1, 2).contiguous()
        self.gate_a_b = self.expect("gate_a.bias", (self.blocks, part)).reshape(-1).contiguous()
        self.gate_i_b = self.expect("gate_i.bias", (self.blocks, part)).reshape(-1).contiguous()
        self.lam = self.expect("lam", (W,))
        self.w_out = self.expect("out.weight", (E, W))
        self.conv_elems = (self.taps - 1) * W
        kernels.mixers()

    def cache_needs(self) -> CacheNeeds:
        return CacheNeeds(state=StateSpec(shape=(self.conv_elems + self.width,), dtype=torch.float32))

    def forward(self, x, ctx, cache):
        T, W = ctx.num_tokens, self.width
        ws = ctx.workspace
        if hasattr(x, "materialize"):
            x = x.materialize()
        proj = ws.get(f"recurrence.in{self.in_width}", (ws.max_tokens, self.in_width), self.dtype)
        linear(x, self.w_in, self.b_in, proj, T, self.b_in_lowp, status=ctx.status)
        u = ws.get(f"recurrence.u{W}", (ws.max_tokens, W), torch.float32)
        state = cache.state
        kernels.conv_tokens(proj[:, W : 2 * W], self.conv_w, self.conv_b, state[:, : max(self.conv_elems, 1)], u,
                            ctx.q_start, ctx.q_len, ctx.seq_slots, ctx.num_seqs, T, kernels.ACT_NONE)
        a = ws.get(f"recurrence.a{W}", (ws.max_tokens, W), torch.float32)
        b = ws.get(f"recurrence.b{W}", (ws.max_tokens, W), torch.float32)
        kernels.rglru_gates(u, self.gate_a_t, self.gate_a_b, self.gate_i_t, self.gate_i_b, self.lam,
                            self.decay_scale, a, b, T, w_a=self.gate_a, w_i=self.gate_i)
        gated = ws.get(f"recurrence.gated{W}", (ws.max_tokens, W), self.dtype)
        scratch = None
        if T > ctx.num_seqs:
            # Portions: long ones run in chunks of tokens side by side.
            size = kernels.rglru_scan_scratch(ws.max_tokens, state.shape[0], W)
            scratch = ws.get(f"recurrence.chunks{W}", (size,), torch.float32)
        kernels.rglru_scan(a, b, proj[:, :W], state[:, self.conv_elems : self.conv_elems + W], gated, ctx.q_start,
                           ctx.q_len, ctx.seq_slots, ctx.num_seqs, self.branch_act, scratch=scratch, num_tokens=T)
        out = ws.get(f"recurrence.out{self.hidden_size}", (ws.max_tokens, self.hidden_size), self.dtype)
        linear(gated, self.w_out, None, out, T, status=ctx.status)
        return out


@register_part("mixer", "state_space")
class StateSpace(Mixer):
    takes_padded_steps = True

    def __init__(self, params, weights, dtype, device, position=None) -> None:
        super().__init__(params, weights, dtype, device)
        self.hidden_size = E = int(params["hidden_size"])
        self.heads = H = int(params["heads"])
        self.value_dim = P = int(params["value_dim"])
        self.state_size = N = int(params["state_size"])
        self.groups = G = int(params["groups"])
        self.norm_groups = int(params.get("norm_groups", 1))
        self.taps = int(params["conv_taps"])
        self.eps = float(params["eps"])
        self.inner = inner = H * P
        if H % G != 0:
            raise ValueError(f"heads={H} is not a multiple of groups={G}")
        if inner % self.norm_groups != 0:
            raise ValueError(f"heads * value_dim = {inner} is not a multiple of norm_groups={self.norm_groups}")
        self.conv_channels = C = inner + 2 * G * N
        rows = 2 * inner + 2 * G * N + H
        self.w_in = _pad_rows(self.expect("in.weight", (rows, E)))
        self.in_width = self.w_in.shape[0]
        self.conv_w = self.expect("conv.weight", (C, self.taps))
        self.conv_b = self.expect("conv.bias", (C,))
        self.dt_bias = self.expect("dt_bias", (H,))
        self.a_log = self.expect("a_log", (H,))
        self.d_skip = self.expect("d", (H,))
        self.norm_w = self.expect("norm.weight", (inner,))
        self.w_out = self.expect("out.weight", (E, inner))
        self.conv_elems = (self.taps - 1) * C
        self.state_elems = H * N * P
        if N > 512:
            raise ValueError(f"state_size={N} is more than the scan kernel holds in a warp's registers (512)")
        kernels.mixers()

    def cache_needs(self) -> CacheNeeds:
        return CacheNeeds(state=StateSpec(shape=(self.conv_elems + self.state_elems,), dtype=torch.float32))

    def forward(self, x, ctx, cache):
        T, inner, C = ctx.num_tokens, self.inner, self.conv_channels
        ws = ctx.workspace
        if hasattr(x, "materialize"):
            x = x.materialize()
        proj = ws.get(f"state_space.in{self.in_width}", (ws.max_tokens, self.in_width), self.dtype)
        linear(x, self.w_in, None, proj, T, status=ctx.status)
        xbc = ws.get(f"state_space.xbc{C}", (ws.max_tokens, C), torch.float32)
        state = cache.state
        kernels.conv_tokens(proj[:, inner : inner + C], self.conv_w, self.conv_b, state[:, : max(self.conv_elems, 1)],
                            xbc, ctx.q_start, ctx.q_len, ctx.seq_slots, ctx.num_seqs, T, kernels.ACT_SILU)
        y = ws.get(f"state_space.y{inner}", (ws.max_tokens, inner), torch.float32)
        scratch = None
        if T > ctx.num_seqs:
            # Portions: long ones run in chunks of tokens side by side.
            size = kernels.ssd_scan_scratch(ws.max_tokens, state.shape[0], self.heads, self.state_size, self.value_dim)
            scratch = ws.get(f"state_space.chunks{self.heads}_{self.state_size}_{self.value_dim}", (size,), torch.float32)
        kernels.ssd_scan(xbc, proj[:, inner + C : inner + C + self.heads], self.dt_bias, self.a_log, self.d_skip,
                         state[:, self.conv_elems : self.conv_elems + self.state_elems], y, self.heads, self.groups,
                         self.state_size, self.value_dim, ctx.q_start, ctx.q_len, ctx.seq_slots, ctx.num_seqs,
                         scratch=scratch, num_tokens=T)
        normed = ws.get(f"state_space.normed{inner}", (ws.max_tokens, inner), self.dtype)
        kernels.gated_group_norm(y, proj[:, :inner], self.norm_w, self.eps, self.norm_groups, normed, T)
        if ctx.residual is not None and self.dtype != torch.float32:
            if use_tensor_core_kernel(normed, self.w_out, T):
                linear(normed, self.w_out, None, ctx.residual, T, status=ctx.status, accumulate=True)
                return None
        out = ws.get(f"state_space.out{self.hidden_size}", (ws.max_tokens, self.hidden_size), self.dtype)
        linear(normed, self.w_out, None, out, T, status=ctx.status)
        return out


@register_part("mixer", "delta_rule")
class DeltaRule(Mixer):
    takes_padded_steps = True

    def __init__(self, params, weights, dtype, device, position=None) -> None:
        super().__init__(params, weights, dtype, device)
        self.hidden_size = E = int(params["hidden_size"])
        self.heads = H = int(params["heads"])
        self.dim = D = int(params["dim"])
        self.eps = float(params["eps"])
        self.decay_scale = float(params["decay_scale"])
        self.key_eps = float(params.get("key_eps", 1e-6))
        self.decay_rank = R = int(params["decay_rank"])
        if D > 512:
            raise ValueError(f"dim={D} is more than the scan kernel holds in a column's lanes (512)")
        self.inner = inner = H * D
        # r | k | v | g | a | w1 in one projection.  W_w1 is followed by rows of zeros up to a
        # multiple of eight, so tanh(W_w1 x) comes out padded with zeros to whole 16-byte rows; the
        # matching columns of W_w2 are zero.
        self.rank_padded = -(-R // 8) * 8
        w_in = self.expect("in.weight", (5 * inner + R, E))
        if self.rank_padded != R:
            w_in = torch.cat([w_in, w_in.new_zeros(self.rank_padded - R, E)])
        self.w_in = _pad_rows(w_in)
        self.in_width = self.w_in.shape[0]
        w2 = self.expect("decay_up.weight", (inner, R))
        if self.rank_padded != R:
            w2 = torch.cat([w2, w2.new_zeros(inner, self.rank_padded - R)], dim=1)
        self.w_decay_up = w2.contiguous()
        self.decay_bias = self.expect("decay_bias", (inner,))
        self.removal_bias = self.expect("removal_bias", (inner,))
        self.norm_w = self.expect("norm.weight", (inner,))
        self.w_out = self.expect("out.weight", (E, inner))
        self.state_elems = H * D * D
        kernels.mixers()

    def cache_needs(self) -> CacheNeeds:
        return CacheNeeds(state=StateSpec(shape=(self.state_elems,), dtype=torch.float32))

    def forward(self, x, ctx, cache):
        T, inner = ctx.num_tokens, self.inner
        ws = ctx.workspace
        if hasattr(x, "materialize"):
            x = x.materialize()
        proj = ws.get(f"delta_rule.in{self.in_width}", (ws.max_tokens, self.in_width), self.dtype)
        linear(x, self.w_in, None, proj, T, status=ctx.status)
        # The decay's logits: the second small matrix on the tanh of the first one's product.
        bent = ws.get(f"delta_rule.bent{self.rank_padded}", (ws.max_tokens, self.rank_padded), self.dtype)
        kernels.act_rows(proj[:, 5 * inner : 5 * inner + self.rank_padded], bent, T, kernels.ACT_TANH)
        logits = ws.get(f"delta_rule.decay{inner}", (ws.max_tokens, inner), self.dtype)
        linear(bent, self.w_decay_up, None, logits, T, status=ctx.status)
        y = ws.get(f"delta_rule.y{inner}", (ws.max_tokens, inner), torch.float32)
        width = kernels.delta_rule_packed_width(self.heads, self.dim, self.dim)
        packed = ws.get(f"delta_rule.packed{width}", (ws.max_tokens, width), torch.float32)
        scratch = None
        if T >= 512:
            # Long steps: chunks of tokens side by side.
            size = kernels.delta_rule_chunk_scratch(ws.max_tokens, cache.state.shape[0], self.heads, self.dim, self.dim)
            scratch = ws.get(f"delta_rule.chunks{self.heads}_{self.dim}", (size,), torch.float32)
        kernels.delta_rule_scan(
            proj[:, :inner], proj[:, inner : 2 * inner], proj[:, 2 * inner : 3 * inner],
            proj[:, 4 * inner : 5 * inner], logits, self.decay_bias, self.removal_bias, self.decay_scale,
            self.key_eps, cache.state, y, self.heads, self.dim, self.dim, ctx.q_start, ctx.q_len, ctx.seq_slots,
            ctx.num_seqs, T, packed, ctx.status, chunk_scratch=scratch)
        normed = ws.get(f"delta_rule.normed{inner}", (ws.max_tokens, inner), self.dtype)
        kernels.gated_group_norm(y, proj[:, 3 * inner : 4 * inner], self.norm_w, self.eps, self.heads, normed, T,
                                 gate_after=True)
        out = ws.get(f"delta_rule.out{self.hidden_size}", (ws.max_tokens, self.hidden_size), self.dtype)
        linear(normed, self.w_out, None, out, T, status=ctx.status)
        return out


@register_part("mixer", "gated_delta_rule")
class GatedDeltaRule(Mixer):
    """``params``: hidden_size, heads, kv_heads, dim, value_dim, conv_taps, eps, unit_eps; ``decay`` ("head",
    "channel"), ``decay_rank`` (0: the logits are rows of the first projection); ``gate_activation``
    ("silu", "sigmoid"), ``gate_rank``.  ``in.weight`` holds the rows q | k | v | b | a | g, with a (g) the
    first half of its low-rank pair where there is one; the second halves are ``decay_up.weight`` and
    ``gate_up.weight``; ``conv.weight`` [channels of q | k | v, taps]."""

    takes_padded_steps = True
    takes_residual_scale = True
    accepts_pending_norm = True

    # Steps of so many tokens and more run their portions in chunks of matrix products; shorter ones, and
    # key sizes the chunks do not take, token after token (from SIDE_BY_SIDE_TOKENS on in long chunks side
    # by side).
    CHUNKED_FROM_TOKENS = 64
    SIDE_BY_SIDE_TOKENS = 512

    def __init__(self, params, weights, dtype, device, position=None) -> None:
        super().__init__(params, weights, dtype, device)
        self.hidden_size = E = int(params["hidden_size"])
        self.heads = H = int(params["heads"])
        self.kv_heads = G = int(params["kv_heads"])
        self.dim = D = int(params["dim"])
        self.value_dim = V = int(params["value_dim"])
        self.taps = int(params["conv_taps"])
        self.eps = float(params["eps"])
        self.unit_eps = float(params.get("unit_eps", 1e-6))
        if H % G:
            raise ValueError(f"heads={H} is not a multiple of kv_heads={G}")
        if D > 512:
            raise ValueError(f"dim={D} is more than the kernels hold in a column's lanes (512)")
        if self.taps < 1:
            raise ValueError("conv_taps must be at least 1")
        if params.get("decay", "head") not in ("head", "channel"):
            raise ValueError(f"gated_delta_rule: decay is 'head' or 'channel', not {params.get('decay')!r}")
        self.per_channel = params.get("decay", "head") == "channel"
        self.gate_act = {"sigmoid": kernels.GATE_SIGMOID, "silu": kernels.GATE_SILU}[params.get("gate_activation", "silu")]
        self.decay_rank, self.gate_rank = int(params.get("decay_rank") or 0), int(params.get("gate_rank") or 0)
        if self.decay_rank and not self.per_channel:
            raise ValueError("gated_delta_rule: a low-rank decay is a decay per channel")
        self.q_scale = D ** -0.5
        self.inner = inner = H * V
        self.channels = C = 2 * G * D + inner
        a_rows = self.decay_rank or (H * D if self.per_channel else H)
        g_rows = self.gate_rank or inner
        w_in = self.expect("in.weight", (C + H + a_rows + g_rows, E))
        # Columns of the first product: q | k | v | b, padding to whole 16-byte packs, a | g.  The low-rank
        # pairs' inner columns then make one aligned range (with zeros behind it) for the second product.
        self.b_at = C
        self.a_at = -(-(C + H) // 8) * 8
        self.g_at = self.a_at + a_rows
        self.in_width = -(-(self.g_at + g_rows) // 8) * 8
        wide = w_in.new_zeros(self.in_width, E)
        wide[: C + H] = w_in[: C + H]
        wide[self.a_at : self.g_at + g_rows] = w_in[C + H :]
        self.w_in = wide
        self.weights.pop("in.weight", None)
        self.conv_t = self.expect("conv.weight", (C, self.taps)).to(torch.float32).t().contiguous()
        self.a_log = self.expect("a_log", (H,))
        self.dt_bias = self.expect("dt_bias", (H * D if self.per_channel else H,))
        self.norm_w = self.expect("norm.weight", (V,))
        self.norm_all = self.norm_w.repeat(H).contiguous()
        self.w_out = self.expect("out.weight", (E, inner))
        self.w_decay_up = self.expect("decay_up.weight", (H * D, self.decay_rank)).contiguous() if self.decay_rank else None
        self.w_gate_up = self.expect("gate_up.weight", (inner, self.gate_rank)).contiguous() if self.gate_rank else None
        self.w_up = None
        if self.decay_rank or self.gate_rank:
            # Both second halves as one product over the inner columns of both pairs.
            start = self.a_at if self.decay_rank else self.g_at
            self.low_at = start // 8 * 8
            self.low_width = self.in_width - self.low_at if self.gate_rank else -(-(self.g_at - self.low_at) // 8) * 8
            self.up_a_rows = H * D if self.decay_rank else 0
            up = wide.new_zeros(self.up_a_rows + (inner if self.gate_rank else 0), self.low_width)
            if self.decay_rank:
                up[: self.up_a_rows, self.a_at - self.low_at : self.a_at - self.low_at + self.decay_rank] = self.w_decay_up
            if self.gate_rank:
                at = self.g_at - self.low_at
                up[self.up_a_rows :, at : at + self.gate_rank] = self.w_gate_up
            self.w_up = up.contiguous()
        self.state_elems = -(-H * V * D // 4) * 4
        self.ring_elems = self.taps * C if self.taps > 1 else 0
        kernels.mixers()

    def cache_needs(self) -> CacheNeeds:
        return CacheNeeds(state=StateSpec(shape=(-(-(self.state_elems + self.ring_elems) // 4) * 4,), dtype=torch.float32))

    def forward(self, x, ctx, cache):
        T, H, G, D, V, C, inner = (ctx.num_tokens, self.heads, self.kv_heads, self.dim, self.value_dim, self.channels,
                                   self.inner)
        ws = ctx.workspace
        proj = ws.get(f"gated_delta.in{self.in_width}", (ws.max_tokens, self.in_width), self.dtype)
        linear(x, self.w_in, None, proj, T, status=ctx.status)
        state = cache.state[:, : self.state_elems]
        ring = cache.state[:, self.state_elems :] if self.taps > 1 else state
        normed = ws.get(f"gated_delta.normed{inner}", (ws.max_tokens, inner), self.dtype)
        a = proj[:, self.a_at : self.g_at]
        g = proj[:, self.g_at : self.g_at + (self.gate_rank or inner)]
        b = proj[:, self.b_at : self.b_at + H]
        rule = (self.per_channel, self.dt_bias, self.a_log, self.conv_t, ring, state, ctx.positions, self.unit_eps,
                self.q_scale, H, G, D, V)
        done = ctx.single_tokens and kernels.gated_delta_step(
            proj[:, :C], b, a, *rule, g, self.norm_w, self.eps, self.gate_act, normed, ctx.q_start, ctx.seq_slots,
            ctx.num_seqs, a_up=self.w_decay_up, g_up=self.w_gate_up)
        if not done:
            if self.w_up is not None:
                low = ws.get(f"gated_delta.low{self.low_width}", (ws.max_tokens, self.low_width), self.dtype)
                kernels.act_rows(proj[:, self.low_at : self.low_at + self.low_width], low, T, kernels.ACT_NONE)
                up = ws.get(f"gated_delta.up{self.w_up.shape[0]}", (ws.max_tokens, self.w_up.shape[0]), self.dtype)
                linear(low, self.w_up, None, up, T, status=ctx.status)
                a = up[:, : self.up_a_rows] if self.decay_rank else a
                g = up[:, self.up_a_rows :] if self.gate_rank else g
            y = ws.get(f"gated_delta.y{inner}", (ws.max_tokens, inner), torch.float32)
            self._recur(proj[:, :C], b, a, rule, y, ctx, cache, T)
            kernels.gated_group_norm(y, g, self.norm_all, self.eps, H, normed, T, gate_after=self.gate_act)
        if (ctx.residual is not None and ctx.status is not None and self.dtype != torch.float32
                and use_tensor_core_kernel(normed, self.w_out, T)):
            linear(normed, self.w_out, None, ctx.residual, T, status=ctx.status, accumulate=True, scale=ctx.residual_scale)
            return None
        out = ws.get("mixer.out", (ws.max_tokens, self.hidden_size), self.dtype)
        linear(normed, self.w_out, None, out, T, status=ctx.status)
        return out


    def _recur(self, x, b, a, rule, y, ctx, cache, T) -> None:
        ws = ctx.workspace
        H, D, V = self.heads, self.dim, self.value_dim
        if T >= self.CHUNKED_FROM_TOKENS:
            size = kernels.gated_delta_chunk_scratch(ws.max_tokens, cache.state.shape[0], H, D, V)
            if size > 0:
                records = ws.get("gated_delta.records%d" % size, (size,), torch.float32)
                if kernels.gated_delta_chunks(x, b, a, *rule, y, ctx.q_start, ctx.q_len, ctx.seq_slots, ctx.num_seqs, T,
                                              records, ctx.status):
                    return
        width = kernels.gated_delta_packed_width(self.per_channel, H, D, V)
        packed = ws.get(f"gated_delta.packed{width}", (ws.max_tokens, width), torch.float32)
        scratch = None
        if T >= self.SIDE_BY_SIDE_TOKENS:
            size = kernels.delta_rule_chunk_scratch(ws.max_tokens, cache.state.shape[0], H, D, V)
            scratch = ws.get(f"gated_delta.chunks{H}_{D}_{V}", (size,), torch.float32)
        kernels.gated_delta_scan(x, b, a, *rule, y, ctx.q_start, ctx.q_len, ctx.seq_slots, ctx.num_seqs, T, packed,
                                 ctx.status, chunk_scratch=scratch)


@register_part("mixer", "selective_scan")
class SelectiveScan(Mixer):
    """``params``: hidden_size, inner, state_size, rank, conv_taps.  ``in.weight`` holds the rows x | z, ``low.weight`` the
    rows low | B | C.  A request's state row holds S as [channel][state], then the convolution's last inputs."""

    takes_padded_steps = True

    def __init__(self, params, weights, dtype, device, position=None) -> None:
        super().__init__(params, weights, dtype, device)
        self.hidden_size = E = int(params["hidden_size"])
        self.inner = I = int(params["inner"])
        self.state_size = N = int(params["state_size"])
        self.rank = R = int(params["rank"])
        self.taps = int(params["conv_taps"])
        if N > 512:
            raise ValueError(f"state_size={N} is more than the scan kernel holds of a channel (512)")
        if self.taps < 1:
            raise ValueError("conv_taps must be at least 1")
        # x | z, each padded with rows of zeros to whole 16-byte packs.
        self.inner_padded = P = -(-I // 8) * 8
        w_in = self.expect("in.weight", (2 * I, E))
        self.w_in = torch.cat([_pad_rows(w_in[:I]), _pad_rows(w_in[I:])]).contiguous()
        self.w_low = _pad_cols(_pad_rows(self.expect("low.weight", (R + 2 * N, I))))
        self.low_width = self.w_low.shape[0]
        self.w_dt = self.expect("dt.weight", (I, R)).contiguous()
        # As a product of its own it reads whole rows of low, B and C against columns of zeros.
        self.w_dt_wide = _pad_rows(_pad_cols(self.w_dt, self.low_width))
        self.weights.pop("in.weight", None)
        self.conv_t = self.expect("conv.weight", (I, self.taps)).to(torch.float32).t().contiguous()
        self.conv_b = self.expect("conv.bias", (I,)).to(torch.float32).contiguous()
        self.dt_bias = self.expect("dt.bias", (I,)).to(torch.float32).contiguous()
        # A log2(e), formed once: the kernels' exponentials are powers of two.
        a = -torch.exp(self.expect("a_log", (I, N)).to(torch.float64))
        self.a2 = (a * math.log2(math.e)).to(torch.float32).contiguous()
        self.d_skip = self.expect("d", (I,)).to(torch.float32).contiguous()
        self.w_out = _pad_cols(self.expect("out.weight", (E, I)))
        self.state_elems = -(-I * N // 4) * 4
        self.conv_elems = (self.taps - 1) * I
        kernels.mixers()

    def cache_needs(self) -> CacheNeeds:
        return CacheNeeds(state=StateSpec(shape=(-(-(self.state_elems + self.conv_elems) // 4) * 4,), dtype=torch.float32))

    def forward(self, x, ctx, cache):
        T, I, P, R, N = ctx.num_tokens, self.inner, self.inner_padded, self.rank, self.state_size
        ws = ctx.workspace
        if hasattr(x, "materialize"):
            x = x.materialize()
        proj = ws.get(f"selective.in{2 * P}", (ws.max_tokens, 2 * P), self.dtype)
        linear(x, self.w_in, None, proj, T, status=ctx.status)
        # (Columns behind I stay zero in both buffers: nothing writes them.)
        u = ws.get(f"selective.x{I}_{P}", (ws.max_tokens, P), self.dtype)
        state = cache.state
        conv_state = state[:, self.state_elems :] if self.taps > 1 else state
        kernels.conv_act(proj[:, :I], self.conv_t, self.conv_b, conv_state, u[:, :I], ctx.q_start, ctx.q_len, ctx.seq_slots,
                         ctx.num_seqs, T, kernels.ACT_SILU)
        low = ws.get(f"selective.low{self.low_width}", (ws.max_tokens, self.low_width), self.dtype)
        linear(u, self.w_low, None, low, T, status=ctx.status)
        y = ws.get(f"selective.y{I}_{P}", (ws.max_tokens, P), self.dtype)
        z = proj[:, P : P + I]
        done = ctx.single_tokens and kernels.selective_step(
            u[:, :I], low, self.w_dt, self.dt_bias, self.a2, self.d_skip, z, y[:, :I], state[:, : self.state_elems],
            ctx.q_start, ctx.seq_slots, ctx.num_seqs)
        if not done:
            dt = ws.get(f"selective.dt{P}", (ws.max_tokens, P), torch.float32)
            linear(low, self.w_dt_wide, None, dt, T, status=ctx.status)
            chunk = kernels.selective_chunk(T, ctx.num_seqs, I, N)
            chunk_states = chunk_dt = None
            if chunk:
                # Places for the chunks (of at least 64 tokens) of any step.
                places = ws.max_tokens // 64 + state.shape[0] + 1
                chunk_states = ws.get(f"selective.chunk_states{I}_{N}", (places * I * N,), torch.float32)
                chunk_dt = ws.get(f"selective.chunk_dt{I}", (places * I,), torch.float32)
            kernels.selective_scan(u[:, :I], dt[:, :I], self.dt_bias, self.a2, low[:, R : R + 2 * N], self.d_skip, z, y[:, :I],
                                   state[:, : self.state_elems], ctx.q_start, ctx.q_len, ctx.seq_slots, ctx.num_seqs, T, ctx.status,
                                   chunk=chunk, chunk_states=chunk_states, chunk_dt=chunk_dt)
        return product_of(y, self.w_out, ctx, T)


@register_part("mixer", "gated_linear_attention")
class GatedLinearAttention(Mixer):
    """``params``: hidden_size, heads, dim, value_dim, rank, tau, eps.  ``in.weight`` holds the rows q | k | v | g | low; the
    second half of the decay's low-rank pair is ``decay_up.weight`` with ``decay_bias``.  A request's state row holds S
    as [head][value][key]."""

    takes_padded_steps = True

    def __init__(self, params, weights, dtype, device, position=None) -> None:
        super().__init__(params, weights, dtype, device)
        self.hidden_size = E = int(params["hidden_size"])
        self.heads = H = int(params["heads"])
        self.dim = D = int(params["dim"])
        self.value_dim = V = int(params["value_dim"])
        self.rank = R = int(params["rank"])
        self.tau = float(params["tau"])
        self.eps = float(params["eps"])
        if D > 512:
            raise ValueError(f"dim={D} is more than the kernels hold in a column's lanes (512)")
        if not self.tau > 0.0:
            raise ValueError(f"tau={self.tau} must be positive")
        self.q_scale = D ** -0.5
        keys, inner = H * D, H * V
        self.inner, self.inner_padded = inner, -(-inner // 8) * 8
        # q | k | v, padding to whole packs, g | low.
        w = self.expect("in.weight", (2 * keys + 2 * inner + R, E))
        self.g_at = -(-(2 * keys + inner) // 8) * 8
        self.low_at = -(-(self.g_at + inner) // 8) * 8
        self.rank_padded = -(-R // 8) * 8
        wide = w.new_zeros(self.low_at + self.rank_padded, E)
        wide[: 2 * keys + inner] = w[: 2 * keys + inner]
        wide[self.g_at : self.g_at + inner] = w[2 * keys + inner : 2 * keys + 2 * inner]
        wide[self.low_at : self.low_at + R] = w[2 * keys + 2 * inner :]
        self.w_in = wide
        self.in_width = wide.shape[0]
        self.weights.pop("in.weight", None)
        self.w_up = self.expect("decay_up.weight", (keys, R)).contiguous()
        self.w_up_wide = _pad_rows(_pad_cols(self.w_up))
        self.decay_bias = self.expect("decay_bias", (keys,)).to(torch.float32).contiguous()
        self.norm_w = self.expect("norm.weight", (V,)).to(torch.float32).contiguous()
        self.norm_all = self.norm_w.repeat(H).contiguous()
        self.w_out = _pad_cols(self.expect("out.weight", (E, inner)))
        self.state_elems = -(-H * V * D // 4) * 4
        kernels.mixers()

    def cache_needs(self) -> CacheNeeds:
        return CacheNeeds(state=StateSpec(shape=(self.state_elems,), dtype=torch.float32))

    def forward(self, x, ctx, cache):
        T, H, D, V, R = ctx.num_tokens, self.heads, self.dim, self.value_dim, self.rank
        keys, inner = H * D, self.inner
        ws = ctx.workspace
        if hasattr(x, "materialize"):
            x = x.materialize()
        proj = ws.get(f"gated_linear.in{self.in_width}", (ws.max_tokens, self.in_width), self.dtype)
        linear(x, self.w_in, None, proj, T, status=ctx.status)
        q, k, v = proj[:, :keys], proj[:, keys : 2 * keys], proj[:, 2 * keys : 2 * keys + inner]
        g = proj[:, self.g_at : self.g_at + inner]
        # (Columns behind inner stay zero: nothing writes them.)
        normed = ws.get(f"gated_linear.normed{inner}", (ws.max_tokens, self.inner_padded), self.dtype)
        state = cache.state
        done = ctx.single_tokens and kernels.gated_linear_step(
            q, k, v, proj[:, self.low_at : self.low_at + R], self.w_up, self.decay_bias, self.q_scale, self.tau, H, D, V, g,
            self.norm_w, self.eps, normed[:, :inner], state, ctx.q_start, ctx.seq_slots, ctx.num_seqs)
        if not done:
            low = proj[:, self.low_at : self.low_at + self.rank_padded]
            if self.dtype == torch.float32 or T <= SMALL_STEP_TOKENS:
                # (The library's product takes rows with a pitch.)
                rows = ws.get(f"gated_linear.low{self.rank_padded}", (ws.max_tokens, self.rank_padded), self.dtype)
                kernels.act_rows(low, rows, T, kernels.ACT_NONE)
                low = rows
            z = ws.get(f"gated_linear.z{self.w_up_wide.shape[0]}", (ws.max_tokens, self.w_up_wide.shape[0]), torch.float32)
            linear(low, self.w_up_wide, None, z, T, status=ctx.status)
            size = kernels.gated_linear_scratch(ws.max_tokens, state.shape[0], H, D)
            records = ws.get("gated_linear.records%d" % size, (size,), torch.float32)
            y = ws.get(f"gated_linear.y{inner}", (ws.max_tokens, inner), torch.float32)
            kernels.gated_linear_chunks(q, k, v, z[:, :keys], self.decay_bias, self.q_scale, self.tau, H, D, V, records, state,
                                        y, ctx.q_start, ctx.q_len, ctx.seq_slots, ctx.num_seqs, T, ctx.status)
            kernels.gated_group_norm(y, g, self.norm_all, self.eps, H, normed[:, :inner], T, gate_after=kernels.GATE_SILU)
        return product_of(normed, self.w_out, ctx, T)


@register_part("mixer", "side_by_side")
class SideBySide(Mixer):
    """Two mixers on the same input.  ``params``: ``left`` and ``right``, each {kind, params};
    the weights of each child carry its prefix (``left.``, ``right.``); ``left.out_norm`` and
    ``right.out_norm`` are the weights of the RMS norms on the children's results; ``scale``
    (0.5: half the sum), ``eps``.  With ``join`` = "weighted_sum" there are no norms and the
    result is ``left_scale * left + right_scale * right``, summed in float32.  The children's
    caches are this part's: pages from the one, a state row from the other."""

    takes_padded_steps = True

    def __init__(self, params, weights, dtype, device, position=None) -> None:
        super().__init__(params, weights, dtype, device)
        self.hidden_size = int(params["hidden_size"])
        self.join = params.get("join", "normed_mean")
        if self.join not in ("normed_mean", "weighted_sum"):
            raise ValueError(f"side_by_side: join is 'normed_mean' or 'weighted_sum', not {self.join!r}")
        self.weighted = self.join == "weighted_sum"
        self.eps = float(params.get("eps", 0.0))
        self.scale = float(params.get("scale", 0.5))
        self.left_scale = float(params.get("left_scale", 1.0))
        self.right_scale = float(params.get("right_scale", 1.0))
        self.children = []
        for side in ("left", "right"):
            child = params[side]
            own = {name[len(side) + 1:]: t for name, t in weights.items()
                   if name.startswith(side + ".") and name != f"{side}.out_norm"}
            cls = part_class("mixer", child["kind"])
            self.children.append(cls(child["params"], own, dtype, device, position=position))
        if self.weighted:
            self.norm_left = self.norm_right = None
            kernels.heads()
        else:
            self.norm_left = self.expect("left.out_norm", (self.hidden_size,))
            self.norm_right = self.expect("right.out_norm", (self.hidden_size,))
        needs = [c.cache_needs() for c in self.children]
        if sum(n.paged is not None for n in needs) > 1 or sum(n.state is not None for n in needs) > 1:
            raise ValueError("side_by_side: at most one child may keep pages and at most one a state")
        self._needs = CacheNeeds(paged=next((n.paged for n in needs if n.paged is not None), None),
                                 state=next((n.state for n in needs if n.state is not None), None))
        self.takes_padded_steps = all(getattr(c, "takes_padded_steps", False) for c in self.children)
        kernels.mixers()

    def cache_needs(self) -> CacheNeeds:
        return self._needs

    def attention_signature(self):
        for child in self.children:
            signature = child.attention_signature()
            if signature is not None:
                return signature
        return None

    def forward(self, x, ctx, cache):
        T = ctx.num_tokens
        if hasattr(x, "materialize"):
            x = x.materialize()
        # The children's results are normed before they join the stream: they must not add
        # into it themselves.
        stream, ctx.residual = ctx.residual, None
        left = self.children[0].forward(x, ctx, cache)
        right = self.children[1].forward(x, ctx, cache)
        ctx.residual = stream
        if self.weighted:
            if stream is not None:
                kernels.add_rows(stream, left, right, T, self.left_scale, self.right_scale)
                return None
            sums = ctx.workspace.get("side_by_side.sums", (ctx.workspace.max_tokens, self.hidden_size), torch.float32)
            sums[:T].zero_()
            kernels.add_rows(sums, left, right, T, self.left_scale, self.right_scale)
            return _lowered_rows(sums, ctx.workspace, self.dtype, T)
        if stream is not None:
            kernels.dual_norm_mean(left, right, self.norm_left, self.norm_right, self.eps, self.scale, T,
                                   resid=stream)
            return None
        out = ctx.workspace.get("side_by_side.out", (ctx.workspace.max_tokens, self.hidden_size), self.dtype)
        kernels.dual_norm_mean(left, right, self.norm_left, self.norm_right, self.eps, self.scale, T, out=out)
        return out
