"""The gated delta rule with a decay per key channel, and with one per head: recurrent mixers whose states live in the cache
manager's slots."""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import LayerCache, Mixer, SharedProjections, StateRequest
from .linear import GEMM_MODULES, linear, linear_sliced
from .registry import norm_class, register_mixer
from .spec import VECTOR, GatedDeltaSpec, HeadDecayDeltaSpec, WeightDecl


class GatedDelta(Mixer):
    """One packed projection [q | k | v | beta | decay's low rank | gate's low rank] -> the short convolution and silu
    of q, k, v (float32 out) -> the two low-rank up-projections (the decay's into float32) -> a pass over the tokens that
    makes q and k unit vectors, exponentiates the decays and takes beta through its sigmoid, and the recurrence over each
    sequence's new tokens (csrc/recurrent.cu: `delta_scan`, two launches) -> RMSNorm of each head's output times sigmoid(gate), one kernel ->
    output projection.

    State of a request, one float32 row of the cache manager's slots: [S (heads x key_dim x value_dim) | the
    convolution's last taps - 1 inputs over the channels of q, k, v side by side, oldest first].  Lengths and slots
    are read from the step's device arrays; any step may be replayed from the graph of its shape."""

    step_arrays_follow_shapes = True
    replay_any_step = True

    @staticmethod
    def weight_decls(spec: GatedDeltaSpec):
        H, G, D, E, W = spec.num_heads, spec.num_kv_heads, spec.key_dim, spec.value_dim, spec.hidden_size
        widths = (G * D, G * D, H * E)
        decls = [WeightDecl(spec.q_proj, (G * D, W)), WeightDecl(spec.k_proj, (G * D, W)), WeightDecl(spec.v_proj, (H * E, W)),
                 WeightDecl(spec.beta_proj, (H, W)), WeightDecl(spec.decay_down, (spec.decay_rank, W)),
                 WeightDecl(spec.decay_up, (H * D, spec.decay_rank)), WeightDecl(spec.decay_bias, (H * D,), VECTOR),
                 WeightDecl(spec.decay_log, (H,), VECTOR), WeightDecl(spec.gate_down, (spec.gate_rank, W)),
                 WeightDecl(spec.gate_up, (H * E, spec.gate_rank)), WeightDecl(spec.o_proj, (W, H * E))]
        decls += [WeightDecl(n, (w, spec.conv.taps), VECTOR) for n, w in zip(spec.conv_weights, widths)]
        return decls + norm_class(spec.out_norm).weight_decls(spec.out_norm)

    @staticmethod
    def kernel_modules(spec):
        return ("recurrent", "rowwise") + GEMM_MODULES

    def __init__(self, spec: GatedDeltaSpec, weights, dtype, device):
        H, G, D, E = spec.num_heads, spec.num_kv_heads, spec.key_dim, spec.value_dim
        if H % G != 0:
            raise ValueError(f"gated delta rule: {H} heads are not a multiple of {G} key heads")
        if D > 256:
            raise ValueError(f"gated delta rule: key width {D} exceeds 256")
        if spec.conv.channels != 2 * G * D + H * E or not 1 <= spec.conv.taps <= 8 or len(spec.conv_weights) != 3:
            raise ValueError("gated delta rule: one convolution of 1 to 8 taps over the channels of q, k and v")
        if spec.out_norm.kind != "rmsnorm" or spec.out_norm.dim != E or spec.out_norm.weight_offset != 0.0:
            raise ValueError("gated delta rule: the output norm is a plain RMSNorm over a head's values")
        self.spec, self.dtype = spec, dtype
        self.H, self.G, self.D, self.E = H, G, D, E
        self.qkv = spec.conv.channels
        names = (spec.q_proj, spec.k_proj, spec.v_proj, spec.beta_proj, spec.decay_down, spec.gate_down)
        self.w_in = torch.cat([weights.device_tensor(n, dtype, device, keep=False) for n in names], dim=0).contiguous()
        self.beta_off = self.qkv
        self.decay_off = self.beta_off + H
        self.gate_off = self.decay_off + spec.decay_rank
        self.w_decay = weights.device_tensor(spec.decay_up, dtype, device)
        self.w_gate = weights.device_tensor(spec.gate_up, dtype, device)
        self.w_o = weights.device_tensor(spec.o_proj, dtype, device)
        self.conv_w = torch.cat([weights.device_tensor(n, dtype, device, keep=False) for n in spec.conv_weights], dim=0).contiguous()
        self.dt_bias = weights.device_tensor(spec.decay_bias, dtype, device).contiguous()
        self.a_log = weights.device_tensor(spec.decay_log, dtype, device).contiguous()
        self.norm_gain = weights.device_tensor(spec.out_norm.weight, dtype, device)
        self.norm_eps = float(spec.out_norm.eps)
        self.s_size = H * D * E

    def state_request(self) -> StateRequest:
        return StateRequest((self.s_size + (self.spec.conv.taps - 1) * self.qkv,), torch.float32)

    def workspace_bytes(self, tokens: int) -> int:
        elem = 2 if self.dtype == torch.bfloat16 else 4
        he = self.H * self.E
        return tokens * (self.w_in.shape[0] * elem + self.qkv * 4 + self.H * self.D * 4 + he * (4 + 2 * elem)
                         + self.spec.hidden_size * elem) + ops.SLICED_PRODUCT_BYTES

    def forward(self, ctx, x, cache: LayerCache):
        T, ws = ctx.n_tokens, ctx.workspace
        H, G, D, E = self.H, self.G, self.D, self.E
        packed = linear(x, self.w_in, ws.buffer("delta_in", T, self.w_in.shape[0], self.dtype))
        qkv = ws.buffer("delta_qkv", T, self.qkv, torch.float32)
        ops.short_conv(qkv, packed[:, :self.qkv], self.conv_w, cache.state[:, self.s_size:], ctx.cu_q, ctx.state_slots, ctx.n_seqs,
                       activation="silu")
        # the decays' up-projection leaves in float32: what follows it (softplus, exponentials) is 32-bit arithmetic
        decay = linear(packed[:, self.decay_off:self.gate_off], self.w_decay, ws.buffer("delta_decay", T, H * D, torch.float32))
        gate = linear(packed[:, self.gate_off:], self.w_gate, ws.buffer("delta_gate", T, H * E, self.dtype))
        o = ws.buffer("delta_o", T, H * E, torch.float32)
        ops.delta_scan(o, qkv, packed[:, self.beta_off:self.decay_off], decay, self.dt_bias, self.a_log, cache.state, ctx.cu_q,
                       ctx.state_slots, ctx.n_seqs, H, G, D, E, float(self.spec.unit_eps), float(D) ** -0.5,
                       beta_buf=ws.buffer("delta_beta", T, H + G, torch.float32))
        y = ws.buffer("delta_y", T, H * E, self.dtype)
        ops.gated_rmsnorm(y.view(T * H, E), o.view(T * H, E), gate, self.norm_gain, self.norm_eps, heads=H)
        return linear_sliced(ws, "mixer_out", y, self.w_o, self.dtype)


class HeadDecayDelta(Mixer):
    """One packed projection [q | k | v | gate | beta | decay] -> one pass over the tokens: the short convolution and silu of q, k, v, unit
    vectors, beta's sigmoid and the decays (`head_delta_prep`, float32 out) -> the recurrence over each sequence's new tokens, for
    steps of `CHUNKED_ROWS` rows and more chunk by chunk (`head_delta_chunks`), else token by token (`delta_scan_heads`) -> RMSNorm of
    each head's output times silu(gate), one kernel -> output projection.  Single tokens, and steps of up to `STEP_ROWS` rows, do all
    between the two projections in one launch (`head_delta_step`).

    State of a request, one float32 row of the cache manager's slots: [S (heads x key_dim x value_dim) | the
    convolution's last taps - 1 inputs over the channels of q, k, v side by side, oldest first].  Lengths and slots
    are read from the step's device arrays; any step may be replayed from the graph of its shape."""

    step_arrays_follow_shapes = True
    replay_any_step = True
    CHUNKED_ROWS = 256
    STEP_ROWS = 16

    @staticmethod
    def weight_decls(spec: HeadDecayDeltaSpec):
        H, G, D, E, W = spec.num_heads, spec.num_kv_heads, spec.key_dim, spec.value_dim, spec.hidden_size
        widths = (G * D, G * D, H * E)
        decls = [WeightDecl(n, (w, W)) for n, w in zip((spec.q_proj, spec.k_proj, spec.v_proj), widths)]
        decls += [WeightDecl(spec.gate_proj, (H * E, W)), WeightDecl(spec.beta_proj, (H, W)), WeightDecl(spec.decay_proj, (H, W)),
                  WeightDecl(spec.decay_bias, (H,), VECTOR), WeightDecl(spec.decay_log, (H,), VECTOR), WeightDecl(spec.o_proj, (W, H * E))]
        decls += [WeightDecl(n, (w, spec.conv.taps), VECTOR) for n, w in zip(spec.conv_weights, widths)]
        return decls + norm_class(spec.out_norm).weight_decls(spec.out_norm)

    @staticmethod
    def kernel_modules(spec):
        return ("head_delta", "recurrent", "rowwise") + GEMM_MODULES

    def __init__(self, spec: HeadDecayDeltaSpec, weights, dtype, device):
        H, G, D, E = spec.num_heads, spec.num_kv_heads, spec.key_dim, spec.value_dim
        if H % G != 0:
            raise ValueError(f"gated delta rule: {H} heads are not a multiple of {G} key heads")
        if D > 256:
            raise ValueError(f"gated delta rule: key width {D} exceeds 256")
        if spec.conv.channels != 2 * G * D + H * E or not 1 <= spec.conv.taps <= 8 or len(spec.conv_weights) != 3:
            raise ValueError("gated delta rule: one convolution of 1 to 8 taps over the channels of q, k and v")
        if spec.out_norm.kind != "rmsnorm" or spec.out_norm.dim != E or spec.out_norm.weight_offset != 0.0:
            raise ValueError("gated delta rule: the output norm is a plain RMSNorm over a head's values")
        self.spec, self.dtype = spec, dtype
        self.H, self.G, self.D, self.E = H, G, D, E
        self.qkv = spec.conv.channels
        names = (spec.q_proj, spec.k_proj, spec.v_proj, spec.gate_proj, spec.beta_proj, spec.decay_proj)
        self.w_in = torch.cat([weights.device_tensor(n, dtype, device, keep=False) for n in names], dim=0).contiguous()
        self.gate_off = self.qkv
        self.beta_off = self.gate_off + H * E
        self.decay_off = self.beta_off + H
        self.w_o = weights.device_tensor(spec.o_proj, dtype, device)
        self.conv_w = torch.cat([weights.device_tensor(n, dtype, device, keep=False) for n in spec.conv_weights], dim=0).contiguous()
        self.dt_bias = weights.device_tensor(spec.decay_bias, dtype, device).contiguous()
        self.a_log = weights.device_tensor(spec.decay_log, dtype, device).contiguous()
        self.norm_gain = weights.device_tensor(spec.out_norm.weight, dtype, device)
        self.norm_eps = float(spec.out_norm.eps)
        self.s_size = H * D * E
        self.step_usable = ops.head_delta_step_usable(H, G, D, E)

    def state_request(self) -> StateRequest:
        return StateRequest((self.s_size + (self.spec.conv.taps - 1) * self.qkv,), torch.float32)

    def workspace_bytes(self, tokens: int) -> int:
        elem = 2 if self.dtype == torch.bfloat16 else 4
        he = self.H * self.E
        chunks = 4 * ops.head_delta_chunk_floats(tokens, max(1, tokens // 32), self.H, self.G, self.D, self.E)
        return chunks + tokens * ((self.decay_off + self.H) * elem + self.qkv * 4 + (2 * self.H + self.G) * 4 + he * (4 + elem)
                         + self.spec.hidden_size * elem) + ops.SLICED_PRODUCT_BYTES

    # -- what a parallel mixer asks that multiplies with several branches' matrices at once (see `parts.parallel`)
    def shared_projections(self):
        return SharedProjections(self.w_in, self.w_o)

    def drop_projections(self) -> None:
        self.w_in = self.w_o = None

    def scale_output(self, factor: float) -> None:
        self.norm_gain = self.norm_gain * factor

    def forward(self, ctx, x, cache: LayerCache):
        T, ws = ctx.n_tokens, ctx.workspace
        packed = linear(x, self.w_in, ws.buffer("hdelta_in", T, self.w_in.shape[0], self.dtype))
        y = ws.buffer("hdelta_y", T, self.H * self.E, self.dtype)
        self.forward_inner(ctx, packed, cache, y)
        return linear_sliced(ws, "hdelta_out", y, self.w_o, self.dtype)

    def forward_inner(self, ctx, packed, cache: LayerCache, y) -> None:
        """From the packed projection to the rows that the output matrix takes."""
        T, ws = ctx.n_tokens, ctx.workspace
        H, G, D, E = self.H, self.G, self.D, self.E
        if (ctx.pure_decode or T <= self.STEP_ROWS) and self.step_usable:
            ops.head_delta_step(y, packed, self.beta_off, self.decay_off, self.gate_off, self.conv_w, self.dt_bias, self.a_log, self.norm_gain,
                                self.norm_eps, cache.state, ctx.cu_q, ctx.state_slots, ctx.n_seqs, H, G, D, E, float(self.spec.unit_eps))
            return
        qkv = ws.buffer("hdelta_qkv", T, self.qkv, torch.float32)
        gates = ws.buffer("hdelta_gates", T, 2 * H + G, torch.float32)
        ops.head_delta_prep(qkv, gates, packed, self.beta_off, self.decay_off, self.conv_w, self.dt_bias, self.a_log,
                            cache.state[:, self.s_size:] if self.spec.conv.taps > 1 else None, ctx.cu_q, ctx.state_slots, ctx.n_seqs,
                            H, G, D, E, float(self.spec.unit_eps))
        o = ws.buffer("hdelta_o", T, H * E, torch.float32)
        floats = ops.head_delta_chunk_floats(T, ctx.n_seqs, H, G, D, E) if T >= self.CHUNKED_ROWS else 0
        if floats:
            scratch = ws.flat("hdelta_chunks", floats, torch.float32)
            ops.head_delta_chunks(o, qkv, gates, cache.state, ctx.cu_q, ctx.state_slots, scratch, ctx.n_seqs, H, G, D, E)
        else:
            ops.delta_scan_heads(o, qkv, gates, cache.state, ctx.cu_q, ctx.state_slots, ctx.n_seqs, H, G, D, E)
        ops.gated_rmsnorm(y, o.view(T * H, E), packed[:, self.gate_off:self.beta_off], self.norm_gain, self.norm_eps,
                          gate_form="silu", heads=H)


register_mixer("gated_delta", GatedDelta)
register_mixer("head_decay_delta", HeadDecayDelta)
