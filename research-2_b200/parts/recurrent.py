"""Mixers that carry a state of fixed size per request instead of a cache that grows with the sequence:
a matrix memory with exponential gates (mLSTM), retention and decay attention (linear attention with a fixed decay per head), a
state-space layer with a short causal convolution (the recurrence of Mamba-2), the gated delta rule behind short convolutions
and time mixing with a decay per channel (RWKV's). Their state lives in 32-bit floats in the request's state slot, starts at
zero with a sequence's first token and is carried from step to step; prompts, portions and single decoded
tokens run through the same kernels (csrc/kernels/recurrent.cu, state_scan.cu), entry by entry, row by row.

All offer `mix(h, ctx, cache, state)`, the mixer's output [T, D] in float32 without the residual stream,
for an arrangement that joins several mixers, beside the usual `forward`, whose last product adds the stream.
"""

from __future__ import annotations

import torch

from ..kernels import ops
from .base import Runtime, StateSpec, register_mixer
from .util import matrix, vector


@register_mixer("mlstm")
class MatrixMemory:
    """Per head a matrix S [dim x vdim], a normaliser n [dim] and a running maximum m of the gates' logarithms:

        log_i = cap(W_i h + b_i), log_f = logsigmoid(cap(W_f h + b_f)), cap(x) = gate_cap tanh(x / gate_cap)
        m' = max(log_f + m, log_i)
        S' = exp(log_f + m - m') S + exp(log_i - m') k v^T,   n' likewise with k alone
        o  = S'^T q / (max(|n' . q|, exp(-m')) + 1e-6),       q = W_q h dim^-1/2, k = W_k h, v = W_v h

    S, n and m start at zero. Each head's o is divided by its root mean square, the heads are concatenated,
    multiplied by `norm`, by sigmoid(W_g h), and projected by W_o.

    params: n_heads, head_dim, v_head_dim, gate_cap (0: none), norm_eps.
    weights (matrices stored [out, in]): w_q, w_k [H * head_dim, D], w_v, w_gate [H * v_head_dim, D], w_out
    [D, H * v_head_dim], norm [H * v_head_dim], w_i, w_f [H, D], b_i, b_f [H].
    The four wide projections run as one product; the gates' as a 32-bit one of their own."""

    def __init__(self, params: dict, weights: dict, rt: Runtime):
        self.n_heads, self.head_dim, self.v_head_dim = int(params["n_heads"]), int(params["head_dim"]), int(params["v_head_dim"])
        self.gate_cap, self.norm_eps = float(params.get("gate_cap", 0.0)), float(params["norm_eps"])
        self.qk_width, self.v_width = self.n_heads * self.head_dim, self.n_heads * self.v_head_dim
        stacked = [weights["w_q"], weights["w_k"], weights["w_v"], weights["w_gate"]]
        if [w.shape[0] for w in stacked] != [self.qk_width, self.qk_width, self.v_width, self.v_width] or \
                weights["w_out"].shape[1] != self.v_width or weights["w_i"].shape[0] != self.n_heads:
            raise ValueError(f"mlstm: projections {[tuple(w.shape) for w in stacked]} and an output of {tuple(weights['w_out'].shape)} "
                             f"do not fit {self.n_heads} heads of {self.head_dim} x {self.v_head_dim}")
        self.w_in = matrix(torch.cat(stacked, dim=0), rt)
        self.w_out = matrix(weights["w_out"], rt)
        self.norm = vector(weights["norm"], rt)
        self.w_gates = vector(torch.cat([weights["w_i"], weights["w_f"]], dim=0), rt)   # float32: the gates enter the recurrence
        self.b_gates = vector(torch.cat([weights["b_i"], weights["b_f"]], dim=0), rt)
        self._state_floats = None

    cache_spec = None
    capturable = True

    def matrices(self):
        return [self.w_in, self.w_out]

    @property
    def state_spec(self) -> StateSpec:
        if self._state_floats is None:
            self._state_floats = self.n_heads * ops.mlstm_state_floats(self.head_dim, self.v_head_dim)
        return StateSpec((self._state_floats,), torch.float32)

    def _inner(self, h, ctx, state):
        proj = ops.linear(h, self.w_in, None, w_is_nk=True)
        gates = ops.small_linear(h, self.w_gates, self.b_gates)
        a, b = self.qk_width, 2 * self.qk_width
        o = ops.mlstm_scan(proj[:, :a], proj[:, a:b], proj[:, b: b + self.v_width], gates, self.gate_cap, self.head_dim ** -0.5,
                           state, ctx.q_start, ctx.state_slot, ctx.fresh, self.n_heads, self.head_dim, self.v_head_dim)
        return ops.group_norm_gated(o, proj[:, b + self.v_width:], self.norm, self.n_heads, self.norm_eps, False, proj.dtype)

    def mix(self, h, ctx, cache=None, state=None, writes_cache: bool = True):
        return ops.linear(self._inner(h, ctx, state), self.w_out, None, w_is_nk=True, out_dtype=torch.float32)

    def forward(self, h, residual, ctx, cache=None, state=None, writes_cache: bool = True):
        return ops.linear(self._inner(h, ctx, state), self.w_out, None, w_is_nk=True, residual=residual)


@register_mixer("retention")
class Retention:
    """Linear attention with one fixed decay per head and neither softmax nor denominator. Per head:

        S' = decay S + k v^T   (S: [head_dim x v_head_dim], from zero),   o = S'^T q
        q = rotate(W_q h), k = rotate(W_k h) head_dim^-1/2, v = W_v h

    (rotation: of each head the first rot_dims dimensions, dimension i with i + rot_dims / 2, by the angle position *
    rot_freqs[i]). Each head's o is divided by its root mean square (no gain), the heads are concatenated, multiplied by
    silu(W_g h) and projected by W_o. The rotation happens inside the recurrence's kernel, in float32: what enters the
    recurrence is the projections' values and nothing rounded after them.

    params: n_heads, head_dim, v_head_dim, decay (one number per head), rot_dims, rot_freqs, norm_eps.
    weights (stored [out, in], no biases): w_q, w_k [H head_dim, D], w_v, w_gate [H v_head_dim, D], w_out [D, H v_head_dim]."""

    def __init__(self, params: dict, weights: dict, rt: Runtime):
        self.n_heads, self.head_dim, self.v_head_dim = int(params["n_heads"]), int(params["head_dim"]), int(params["v_head_dim"])
        self.norm_eps, self.rot_dims = float(params["norm_eps"]), int(params.get("rot_dims", 0))
        decay, freqs = [float(x) for x in params["decay"]], [float(f) for f in params.get("rot_freqs", ())]
        if len(decay) != self.n_heads or self.rot_dims % 2 or not 0 <= self.rot_dims <= self.head_dim or len(freqs) != self.rot_dims // 2:
            raise ValueError(f"retention: {len(decay)} decays for {self.n_heads} heads, {self.rot_dims} rotated dimensions of "
                             f"{self.head_dim} with {len(freqs)} frequencies")
        self.qk_width, self.v_width = self.n_heads * self.head_dim, self.n_heads * self.v_head_dim
        stacked = [weights["w_q"], weights["w_k"], weights["w_v"], weights["w_gate"]]
        if [w.shape[0] for w in stacked] != [self.qk_width, self.qk_width, self.v_width, self.v_width] or weights["w_out"].shape[1] != self.v_width:
            raise ValueError(f"retention: projections {[tuple(w.shape) for w in stacked]} and an output of {tuple(weights['w_out'].shape)} "
                             f"do not fit {self.n_heads} heads of {self.head_dim} x {self.v_head_dim}")
        self.w_in = matrix(torch.cat(stacked, dim=0), rt)
        self.w_out = matrix(weights["w_out"], rt)
        # decays and frequencies: exact in float64, rounded once to float32
        self.decay = torch.tensor(decay, dtype=torch.float64).to(torch.float32).to(rt.device)
        self.freqs = torch.tensor(freqs, dtype=torch.float64).to(torch.float32).to(rt.device)

    cache_spec = None
    capturable = True

    def matrices(self):
        return [self.w_in, self.w_out]

    @property
    def state_spec(self) -> StateSpec:
        return StateSpec((self.n_heads * self.head_dim * self.v_head_dim,), torch.float32)

    def _inner(self, h, ctx, state):
        proj = ops.linear(h, self.w_in, None, w_is_nk=True)
        a, b = self.qk_width, 2 * self.qk_width
        o = ops.retention_scan(proj[:, :a], proj[:, a:b], proj[:, b: b + self.v_width], self.decay, self.head_dim ** -0.5, self.freqs,
                               self.rot_dims, ctx.positions, state, ctx.q_start, ctx.state_slot, ctx.fresh, self.n_heads, self.head_dim,
                               self.v_head_dim)
        return ops.group_norm_gated(o, proj[:, b + self.v_width:], None, self.n_heads, self.norm_eps, "silu_after", proj.dtype)

    def mix(self, h, ctx, cache=None, state=None, writes_cache: bool = True):
        return ops.linear(self._inner(h, ctx, state), self.w_out, None, w_is_nk=True, out_dtype=torch.float32)

    def forward(self, h, residual, ctx, cache=None, state=None, writes_cache: bool = True):
        return ops.linear(self._inner(h, ctx, state), self.w_out, None, w_is_nk=True, residual=residual)


@register_mixer("decay_attention")
class DecayAttention:
    """Linear attention with one fixed decay per head and silu on queries, keys and values, all heads normed together. Per head:

        S' = decay S + k v^T   (S: [head_dim x v_head_dim], from zero),   o = S'^T q
        q = silu(W_q h), k = silu(W_k h), v = silu(W_v h)

    The concatenated heads are RMS-normed as one row, times `norm`, times sigmoid(W_g h), and projected by W_o. silu is part of the
    recurrence's kernels, in float32: what enters the recurrence is the projections' values. Decoded tokens, and everything in float32, walk
    row by row; prompts in bfloat16 go in chunks of 64 rows on the tensor cores, operands as two bfloat16 terms, the state in float32.

    params: n_heads, head_dim, v_head_dim, decay (one number per head), norm_eps, out_scale (default 1: a factor on the gated outputs,
    folded into the norm's gains).
    weights (stored [out, in], no biases): w_q, w_k [H head_dim, D], w_v, w_gate [H v_head_dim, D], norm [H v_head_dim], w_out
    [D, H v_head_dim]."""

    def __init__(self, params: dict, weights: dict, rt: Runtime):
        self.n_heads, self.head_dim, self.v_head_dim = int(params["n_heads"]), int(params["head_dim"]), int(params["v_head_dim"])
        self.norm_eps, decay = float(params["norm_eps"]), [float(x) for x in params["decay"]]
        self.qk_width, self.inner_width = self.n_heads * self.head_dim, self.n_heads * self.v_head_dim
        stacked = [weights["w_q"], weights["w_k"], weights["w_v"], weights["w_gate"]]
        if (len(decay) != self.n_heads or [w.shape[0] for w in stacked] != [self.qk_width, self.qk_width, self.inner_width, self.inner_width]
                or weights["w_out"].shape[1] != self.inner_width or weights["norm"].shape[0] != self.inner_width):
            raise ValueError(f"decay attention: {len(decay)} decays, projections {[tuple(w.shape) for w in stacked]} and an output of "
                             f"{tuple(weights['w_out'].shape)} do not fit {self.n_heads} heads of {self.head_dim} x {self.v_head_dim}")
        self.w_in = matrix(torch.cat(stacked, dim=0), rt)
        self.w_out = matrix(weights["w_out"], rt)
        self.norm = vector(weights["norm"], rt) * float(params.get("out_scale", 1.0))
        # decays: exact in float64, rounded once to float32
        self.decay = torch.tensor(decay, dtype=torch.float64).to(torch.float32).to(rt.device)

    cache_spec = None
    capturable = True

    def matrices(self):
        return [self.w_in, self.w_out]

    @property
    def state_spec(self) -> StateSpec:
        return StateSpec((self.n_heads * self.head_dim * self.v_head_dim,), torch.float32)

    def input_matrix(self):
        """The stacked projections of the input, [q; k; v; gate] x D stored [out, in], which may run beside another mixer's as one
        product and come back as `proj`."""
        return self.w_in

    def inner(self, h, ctx, cache=None, state=None, writes_cache: bool = True, out=None, proj=None):
        """The gated heads' outputs [T, H v_head_dim] before w_out (into `out` where given)."""
        if proj is None:
            proj = ops.linear(h, self.w_in, None, w_is_nk=True)
        a, b = self.qk_width, 2 * self.qk_width
        o = ops.retention_scan(proj[:, :a], proj[:, a:b], proj[:, b: b + self.inner_width], self.decay, 1.0, None, 0, ctx.positions, state,
                               ctx.q_start, ctx.state_slot, ctx.fresh, self.n_heads, self.head_dim, self.v_head_dim, silu=True,
                               n_tiles=ctx.n_attention_tiles)
        return ops.group_norm_gated(o, proj[:, b + self.inner_width:], self.norm, 1, self.norm_eps, False, proj.dtype, out=out)

    def mix(self, h, ctx, cache=None, state=None, writes_cache: bool = True):
        return ops.linear(self.inner(h, ctx, cache, state), self.w_out, None, w_is_nk=True, out_dtype=torch.float32)

    def forward(self, h, residual, ctx, cache=None, state=None, writes_cache: bool = True):
        return ops.linear(self.inner(h, ctx, cache, state), self.w_out, None, w_is_nk=True, residual=residual)


@register_mixer("ssd")
class StateSpace:
    """inner = n_heads * v_head_dim; W_in h is laid out [z: inner | x: inner | B: groups * n_state | C: groups * n_state |
    dt: n_heads]. x, B and C pass a causal convolution per channel (taps [channels, conv_taps], the last column the
    current token's, zeros before the start) and silu. dt = softplus(dt + dt_bias). Per head (head i uses group
    i // (n_heads / groups)):

        S' = exp(-exp(A_log) dt) S + dt B x^T   (S: [n_state x v_head_dim]),   y = S'^T C + D x

    y (heads concatenated) is multiplied by silu(z), RMS-normed in norm_groups equal parts, times `norm`, then W_o. The
    state is S and the convolution's last conv_taps - 1 inputs.

    params: n_heads, v_head_dim, n_state, n_groups, conv_taps, norm_groups, norm_eps.
    weights: w_in [2 inner + 2 groups n_state + n_heads, D], conv [channels, conv_taps], conv_b [channels], dt_bias, a_log,
    d_skip [n_heads], norm [inner], w_out [D, inner]. The step sizes' rows of w_in run as a 32-bit product of their own."""

    def __init__(self, params: dict, weights: dict, rt: Runtime):
        self.n_heads, self.v_head_dim, self.n_state = int(params["n_heads"]), int(params["v_head_dim"]), int(params["n_state"])
        self.n_groups, self.conv_taps = int(params["n_groups"]), int(params["conv_taps"])
        self.norm_groups, self.norm_eps = int(params["norm_groups"]), float(params["norm_eps"])
        self.inner = self.n_heads * self.v_head_dim
        self.bc_width = self.n_groups * self.n_state
        self.channels = self.inner + 2 * self.bc_width
        w_in = weights["w_in"]
        if w_in.shape[0] != self.inner + self.channels + self.n_heads or tuple(weights["conv"].shape) != (self.channels, self.conv_taps) \
                or weights["w_out"].shape[1] != self.inner or self.n_heads % self.n_groups or self.inner % self.norm_groups:
            raise ValueError(f"ssd: w_in {tuple(w_in.shape)}, conv {tuple(weights['conv'].shape)}, w_out {tuple(weights['w_out'].shape)} do not "
                             f"fit {self.n_heads} heads of {self.v_head_dim}, {self.n_groups} groups of {self.n_state}, {self.conv_taps} taps")
        self.w_in = matrix(w_in[: self.inner + self.channels], rt)
        self.w_steps = vector(w_in[self.inner + self.channels:], rt)
        self.conv, self.conv_b = vector(weights["conv"], rt), vector(weights["conv_b"], rt)
        self.dt_bias, self.a_log, self.d_skip = (vector(weights[k], rt) for k in ("dt_bias", "a_log", "d_skip"))
        self.norm = vector(weights["norm"], rt)
        self.w_out = matrix(weights["w_out"], rt)
        self.conv_state_off = self.n_heads * self.n_state * self.v_head_dim

    cache_spec = None
    capturable = True

    def matrices(self):
        return [self.w_in, self.w_out]

    @property
    def state_spec(self) -> StateSpec:
        return StateSpec((self.conv_state_off + (self.conv_taps - 1) * self.channels,), torch.float32)

    def _inner(self, h, ctx, state):
        proj = ops.linear(h, self.w_in, None, w_is_nk=True)
        steps = ops.small_linear(h, self.w_steps, None)
        z, xbc = proj[:, : self.inner], proj[:, self.inner:]
        mixed = ops.causal_conv(xbc, self.conv, self.conv_b, state, self.conv_state_off, ctx.row_entry, ctx.q_start,
                                ctx.state_slot, ctx.fresh)
        x, b = mixed[:, : self.inner], mixed[:, self.inner: self.inner + self.bc_width]
        y = ops.ssd_scan(x, b, mixed[:, self.inner + self.bc_width:], steps, self.dt_bias, self.a_log, self.d_skip, state,
                         ctx.q_start, ctx.state_slot, ctx.fresh, self.n_heads, self.n_groups, self.n_state, self.v_head_dim,
                         conv_in=xbc, conv_taps=self.conv_taps, conv_state_off=self.conv_state_off)
        return ops.group_norm_gated(y, z, self.norm, self.norm_groups, self.norm_eps, True, proj.dtype)

    def mix(self, h, ctx, cache=None, state=None, writes_cache: bool = True):
        return ops.linear(self._inner(h, ctx, state), self.w_out, None, w_is_nk=True, out_dtype=torch.float32)

    def forward(self, h, residual, ctx, cache=None, state=None, writes_cache: bool = True):
        return ops.linear(self._inner(h, ctx, state), self.w_out, None, w_is_nk=True, residual=residual)


@register_mixer("delta")
class DeltaRule:
    """The gated delta rule: a matrix per head that every row first lets decay, then asks for what it holds under the row's key, and
    then corrects by a share of what is missing. Per head (head i uses the queries and keys of group i // (heads / groups)):

        q, k, v = silu(conv(W_q h)), silu(conv(W_k h)), silu(conv(W_v h))     (a causal convolution per channel, last tap the current row)
        q, k made unit vectors, x / sqrt(sum x^2 + unit_eps); q times head_dim^-1/2
        beta = sigmoid(W_b h), g = exp(-exp(a_log) softplus(W_a h + dt_bias))
        S' = g S, u = beta (v - S'^T k), S = S' + k u^T, o = S^T q            (S: [head_dim x v_head_dim], from zero)

    Each head's o is divided by its root mean square, times `norm` [v_head_dim] (shared by the heads), times silu(W_g h); then W_o. The
    state is S and the convolutions' last conv_taps - 1 inputs. Everything after the
    projections is float32.

    params: n_heads, n_groups, head_dim, v_head_dim, conv_taps, unit_eps, norm_eps.
    weights (stored [out, in], no biases): w_q, w_k [groups head_dim, D], w_v, w_gate [H v_head_dim, D], w_out [D, H v_head_dim], conv_q,
    conv_k [groups head_dim, taps], conv_v [H v_head_dim, taps], w_b, w_a [H, D], a_log, dt_bias [H], norm [v_head_dim].
    The four wide projections run as one product; one launch prepares what the recurrence walks over."""

    def __init__(self, params: dict, weights: dict, rt: Runtime):
        self.n_heads, self.n_groups = int(params["n_heads"]), int(params["n_groups"])
        self.head_dim, self.v_head_dim, self.conv_taps = int(params["head_dim"]), int(params["v_head_dim"]), int(params["conv_taps"])
        self.unit_eps, self.norm_eps = float(params["unit_eps"]), float(params["norm_eps"])
        self.qk_width, self.v_width = self.n_groups * self.head_dim, self.n_heads * self.v_head_dim
        stacked = [weights["w_q"], weights["w_k"], weights["w_v"], weights["w_gate"]]
        convs = [weights["conv_q"], weights["conv_k"], weights["conv_v"]]
        if (self.n_heads % self.n_groups or [w.shape[0] for w in stacked] != [self.qk_width, self.qk_width, self.v_width, self.v_width]
                or [tuple(c.shape) for c in convs] != [(n, self.conv_taps) for n in (self.qk_width, self.qk_width, self.v_width)]
                or weights["w_out"].shape[1] != self.v_width or weights["norm"].shape[0] != self.v_head_dim):
            raise ValueError(f"delta rule: projections {[tuple(w.shape) for w in stacked]}, convolutions {[tuple(c.shape) for c in convs]} and an output of "
                             f"{tuple(weights['w_out'].shape)} do not fit {self.n_heads} heads, {self.n_groups} groups of {self.head_dim} x {self.v_head_dim}")
        self.w_in = matrix(torch.cat(stacked, dim=0), rt)
        self.w_out = matrix(weights["w_out"], rt)
        self.conv = vector(torch.cat(convs, dim=0), rt)
        self.channels = self.conv.shape[0]
        self.w_gates = matrix(torch.cat([weights["w_b"], weights["w_a"]], dim=0), rt)   # (the products with it are float32 sums)
        self.a_log, self.dt_bias = vector(weights["a_log"], rt), vector(weights["dt_bias"], rt)
        self.norm = vector(weights["norm"].repeat(self.n_heads), rt)
        self.conv_state_off = self.n_heads * ops.scan_state_floats(self.head_dim, self.v_head_dim)

    cache_spec = None
    capturable = True

    def matrices(self):
        return [self.w_in, self.w_out]

    @property
    def state_spec(self) -> StateSpec:
        return StateSpec((-(-(self.conv_state_off + (self.conv_taps - 1) * self.channels) // 4) * 4,), torch.float32)   # (whole 16-byte pieces)

    def _inner(self, h, ctx, state):
        proj = ops.linear(h, self.w_in, None, w_is_nk=True)
        raw = proj[:, : self.channels]
        qk, v, numbers = ops.delta_prepare(raw, h, self.conv, self.w_gates, self.dt_bias, self.a_log, self.head_dim ** -0.5, self.unit_eps, self.n_heads,
                                           self.n_groups, self.head_dim, self.v_head_dim, state, self.conv_state_off, ctx.row_entry, ctx.q_start,
                                           ctx.state_slot, ctx.fresh)
        o = ops.delta_scan(qk, v, numbers, self.head_dim, state, ctx.q_start, ctx.state_slot, ctx.fresh, conv_in=raw, conv_taps=self.conv_taps,
                           conv_state_off=self.conv_state_off)
        return ops.group_norm_gated(o, proj[:, self.channels:], self.norm, self.n_heads, self.norm_eps, "silu_after", proj.dtype)

    def mix(self, h, ctx, cache=None, state=None, writes_cache: bool = True):
        return ops.linear(self._inner(h, ctx, state), self.w_out, None, w_is_nk=True, out_dtype=torch.float32)

    def forward(self, h, residual, ctx, cache=None, state=None, writes_cache: bool = True):
        return ops.linear(self._inner(h, ctx, state), self.w_out, None, w_is_nk=True, residual=residual)


@register_mixer("time_mix")
class TimeMix:
    """Time mixing with a decay per channel that depends on the input. h' is the row before h in its sequence (zeros before the first);
    each of r, k, v, g and w reads a mix of its own, mix_s = h + (h' - h) mu_s:

        r, k, v = W_r mix_r, W_k mix_k, W_v mix_v (heads of head_dim); gate = silu(W_g mix_g)
        w = exp(-exp(W_w2 tanh(W_w1 mix_w) + w0))                                   (per head and key channel)
        o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t, then S_t = diag(w_t) S_(t-1) + k_t v_t^T     (S from zero)

    Each head's o is divided by its root mean square, the heads are concatenated, times `norm`, times the gate; then W_o. The state is S
    and the last row h. The way to the decays (mix_w, the sums of both small products, tanh, the exponentials) is float32.

    params: n_heads, head_dim, norm_eps, out_scale (default 1: a factor on the gated outputs, folded into the norm's gains).
    weights (stored [out, in], no biases): w_r, w_k, w_v, w_gate [H head_dim, D], mu_r, mu_k, mu_v, mu_g, mu_w [D], w1 [rank, D], w2 [H head_dim,
    rank], w0 [H head_dim], bonus [H, head_dim], norm [H head_dim], w_out [D, H head_dim]."""

    def __init__(self, params: dict, weights: dict, rt: Runtime):
        self.n_heads, self.head_dim, self.norm_eps = int(params["n_heads"]), int(params["head_dim"]), float(params["norm_eps"])
        self.inner_width = self.n_heads * self.head_dim
        stacked = [weights[n] for n in ("w_r", "w_k", "w_v", "w_gate")]
        self.width = stacked[0].shape[1]
        w1, w2 = weights["w1"], weights["w2"]
        if (any(tuple(w.shape) != (self.inner_width, self.width) for w in stacked) or w1.shape[1] != self.width or w1.shape[0] != w2.shape[1]
                or w2.shape[0] != self.inner_width or weights["w_out"].shape[1] != self.inner_width or weights["bonus"].numel() != self.inner_width):
            raise ValueError(f"time mixing: projections {[tuple(w.shape) for w in stacked]}, decay {tuple(w1.shape)} and {tuple(w2.shape)} and an output of "
                             f"{tuple(weights['w_out'].shape)} do not fit {self.n_heads} heads of {self.head_dim}")
        # [4 groups of H head_dim rows, D]: the rows of each kind read a mix of their own; for the tensor cores a group is padded with
        # zeros to whole tiles, so that the four products are one launch
        self.group = -(-self.inner_width // 128) * 128 if rt.dtype == torch.bfloat16 else self.inner_width
        self.w_in = matrix(torch.cat([torch.nn.functional.pad(w, (0, 0, 0, self.group - self.inner_width)) for w in stacked], dim=0), rt)
        self.w_out = matrix(weights["w_out"], rt)
        self.mu = vector(torch.stack([weights["mu_" + s] for s in "rkvgw"]), rt)
        self.w1, self.w2t, self.w0 = matrix(w1, rt), matrix(w2.T, rt), vector(weights["w0"], rt)
        self.bonus = vector(weights["bonus"].reshape(-1), rt)
        self.norm = vector(weights["norm"], rt) * float(params.get("out_scale", 1.0))
        self.row_state_off = self.n_heads * ops.scan_state_floats(self.head_dim, self.head_dim)

    cache_spec = None
    capturable = True

    def matrices(self):
        return [self.w_in, self.w_out]

    @property
    def state_spec(self) -> StateSpec:
        return StateSpec((-(-(self.row_state_off + self.width) // 4) * 4,), torch.float32)

    def inner(self, h, ctx, cache=None, state=None, writes_cache: bool = True, out=None):
        """The gated heads' outputs [T, H head_dim] before w_out (into `out` where given)."""
        mixes, decay = ops.time_mix_prepare(h, self.mu, self.w1, self.w2t, self.w0, state, self.row_state_off, ctx.row_entry, ctx.q_start,
                                                ctx.state_slot, ctx.fresh)
        proj = ops.grouped_linear(mixes, self.w_in)
        r, k, v, gate = (proj[:, i * self.group: i * self.group + self.inner_width] for i in range(4))
        o = ops.time_mix_scan(r, k, v, decay, self.bonus, state, ctx.q_start, ctx.state_slot, ctx.fresh, self.n_heads, self.head_dim,
                              row_in=h, row_state_off=self.row_state_off)
        return ops.group_norm_gated(o, gate, self.norm, self.n_heads, self.norm_eps, "silu_after", proj.dtype, out=out)

    def mix(self, h, ctx, cache=None, state=None, writes_cache: bool = True):
        return ops.linear(self.inner(h, ctx, cache, state), self.w_out, None, w_is_nk=True, out_dtype=torch.float32)

    def forward(self, h, residual, ctx, cache=None, state=None, writes_cache: bool = True):
        return ops.linear(self.inner(h, ctx, cache, state), self.w_out, None, w_is_nk=True, residual=residual)


class _TwoMixers:
    """Two mixers that read the same input; either may keep a per-token cache and either a per-request state, but only one of each."""

    def _make_sides(self, params: dict, weights: dict, rt: Runtime, ask: str, extra=({}, {})):
        from .base import registry

        self.sides = []
        for side, more in zip(("left", "right"), extra):
            spec = params[side]
            own = {name[len(side) + 1:]: t for name, t in weights.items() if name.startswith(side + ".")}
            part = registry("mixer")[spec["kind"]]({**spec["params"], **more}, own, rt)
            if not hasattr(part, ask):
                raise ValueError(f"two mixers side by side: a mixer of kind {spec['kind']!r} has no `{ask}` (its output without the stream)")
            self.sides.append(part)
        for what in ("cache_spec", "state_spec"):
            if sum(getattr(p, what, None) is not None for p in self.sides) > 1:
                raise ValueError(f"two mixers side by side: both have a {what}; a layer has one cache member and one state member")
        self.capturable = all(getattr(p, "capturable", False) for p in self.sides)

    def _of(self, what):
        return next((getattr(p, what) for p in self.sides if getattr(p, what, None) is not None), None)

    @property
    def cache_spec(self):
        return self._of("cache_spec")

    @property
    def state_spec(self):
        return self._of("state_spec")


@register_mixer("side_by_side_sum")
class SideBySideSum(_TwoMixers):
    """left_scale left(h) + right_scale right(h): two mixers read the same input and their scaled outputs are summed. Each mixer hands over
    what it has before its last product (`inner`, with its scale inside, in float32 before it is rounded), side by side in
    one buffer, and ONE product over both output matrices makes the sum. Where both mixers begin with plain products of the input
    (`input_matrix`), those run as one too.

    params: left, right: {"kind": mixer kind, "params": {...}} (mixers that take `out_scale` and offer `inner`); left_scale, right_scale.
    weights: each mixer's own under the prefixes "left." and "right."."""

    def __init__(self, params: dict, weights: dict, rt: Runtime):
        self._make_sides(params, weights, rt, "inner", ({"out_scale": float(params["left_scale"])}, {"out_scale": float(params["right_scale"])}))
        self.w_out = torch.cat([p.w_out for p in self.sides], dim=1).contiguous()
        at = 0
        for p in self.sides:   # the parts keep views into the joint matrix
            p.w_out, at = self.w_out[:, at: at + p.inner_width], at + p.inner_width
        self.w_in = None
        asked = [getattr(p, "input_matrix", lambda: None)() for p in self.sides]
        if all(m is not None for m in asked):
            self.w_in, self.split = torch.cat(asked, dim=0), asked[0].shape[0]
            self.sides[0].w_in, self.sides[1].w_in = self.w_in[: self.split], self.w_in[self.split:]

    def matrices(self):
        return ([self.sides[0].w_in, self.sides[1].w_in] if self.w_in is None else [self.w_in]) + [self.w_out]

    def _inner(self, h, ctx, cache, state, writes_cache):
        # (rows a multiple of eight numbers apart: the attention kernels write pairs, the product reads 16-byte pieces)
        both = torch.empty(h.shape[0], -(-self.w_out.shape[1] // 8) * 8, dtype=h.dtype, device=h.device)[:, : self.w_out.shape[1]]
        projected = ({}, {})
        if self.w_in is not None:   # (rows a multiple of eight numbers apart, as above)
            proj = torch.empty(h.shape[0], -(-self.w_in.shape[0] // 8) * 8, dtype=h.dtype, device=h.device)[:, : self.w_in.shape[0]]
            ops.linear(h, self.w_in, None, w_is_nk=True, out=proj)
            projected = ({"proj": proj[:, : self.split]}, {"proj": proj[:, self.split:]})
        at = 0
        for p, more in zip(self.sides, projected):
            p.inner(h, ctx, cache, state, writes_cache, out=both[:, at: at + p.inner_width], **more)
            at += p.inner_width
        return both

    def mix(self, h, ctx, cache=None, state=None, writes_cache: bool = True):
        return ops.linear(self._inner(h, ctx, cache, state, writes_cache), self.w_out, None, w_is_nk=True, out_dtype=torch.float32)

    def forward(self, h, residual, ctx, cache=None, state=None, writes_cache: bool = True):
        return ops.linear(self._inner(h, ctx, cache, state, writes_cache), self.w_out, None, w_is_nk=True, residual=residual)


@register_mixer("side_by_side")
class SideBySide(_TwoMixers):
    """Two mixers read the same input; each one's output is RMS-normed over the model width with a plain gain of its
    own, and `share` times their sum joins the stream: x + share (norm(left(h)) w_left + norm(right(h)) w_right).

    params: left, right: {"kind": mixer kind, "params": {...}}; eps; share (default 0.5).
    weights: left_out, right_out [D], and each mixer's own weights under the prefixes "left." and "right.".
    Either mixer may keep a per-token cache and either a per-request state, but only one of each."""

    def __init__(self, params: dict, weights: dict, rt: Runtime):
        self.eps, self.share = float(params["eps"]), float(params.get("share", 0.5))
        self._make_sides(params, weights, rt, "mix")
        self.w_left, self.w_right = vector(weights["left_out"], rt), vector(weights["right_out"], rt)

    def matrices(self):
        return [m for p in self.sides for m in p.matrices()]

    def forward(self, h, residual, ctx, cache=None, state=None, writes_cache: bool = True):
        left, right = (p.mix(h, ctx, cache, state, writes_cache) for p in self.sides)
        return ops.pair_norm_add(residual, left, right, self.w_left, self.w_right, self.eps, self.share)
