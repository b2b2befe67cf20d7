"""A state-space recurrence with one decay per token and head (Mamba-2).

    [z | x | B | C | dt] = W_in h         (inner, inner, groups * state, groups * state and heads elements; inner = heads * size)
    x, B, C <- silu(conv(x, B, C)):  conv(v)_t[c] = b[c] + sum_j w[c, j] v_(t - taps + 1 + j)[c], zeros before the start
    dt <- softplus(dt + dt_bias)
    per head h of group h // (heads / groups):  S_t = exp(-exp(A_log_h) dt) S_(t-1) + dt B_t x_t^T,  S before the start = 0
                                                y_t = S_t^T C_t + D_h x_t
    out = W_o ( rms over each of norm_groups equal parts of (y * silu(z)) * w )

What a request carries from token to token is one 32-bit state per slot: the convolution's last inputs in a ring of `taps`
rows (csrc/conv_ring.cuh) and S [heads, state, size].  Step sizes, decays, exponentials, the state, the sums over it, the
gate and the norm are 32-bit (csrc/state_space.cu).  Single tokens update the state in place (in a step of single tokens alone
that kernel does the convolution too); prompt portions are cut into chunks that run side by side and continue from the slot's
state, in bfloat16 on the tensor cores where they take the sizes (csrc/state_space_tc.cu: x, B and C are then rounded to
bfloat16 behind the convolution, in every kind of step).

Parameters: hidden, heads, size, state, groups, norm_groups, taps, norm_eps, and optionally `names`."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights import TensorSpec
from .base import Mixer, StateRequest, register_mixer
from .linear import ACCUM, STORE, linear, prepare_weight


@register_mixer("state_space")
class StateSpace(Mixer):
    graph_safe = True
    takes_deferred_norm = True
    can_store = True
    projects_input = True
    NAMES = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "A_log": "A_log", "D": "D", "norm": "norm",
             "o": "o"}

    def graph_key(self, ctx) -> tuple:
        return ()            # the chunks' number follows from the step's numbers of tokens, single tokens and portions

    @staticmethod
    def _names(params, prefix):
        return {key: prefix + name for key, name in {**StateSpace.NAMES, **params.get("names", {})}.items()}

    @staticmethod
    def _sizes(params):
        return tuple(int(params[k]) for k in ("heads", "size", "state", "groups", "norm_groups", "taps"))

    @staticmethod
    def check_params(params):
        heads, size, states, groups, norm_groups, taps = StateSpace._sizes(params)
        if heads <= 0 or groups <= 0 or heads % groups:
            raise ValueError("state space: groups must divide heads, both positive")
        if not 0 < size <= ops.SSD_MAX_HEAD or not 0 < states <= ops.SSD_MAX_HEAD:
            raise ValueError(f"state space: size and state within 1..{ops.SSD_MAX_HEAD} (what the kernel takes)")
        if norm_groups <= 0 or (heads * size) % norm_groups:
            raise ValueError("state space: norm_groups must divide heads * size")
        if not 1 <= taps <= ops.RING_MAX_TAPS:
            raise ValueError(f"state space: {taps} taps; the kernel takes 1..{ops.RING_MAX_TAPS}")

    @staticmethod
    def tensor_specs(params, prefix):
        heads, size, states, groups, _, taps = StateSpace._sizes(params)
        h, inner = int(params["hidden"]), heads * size
        n, conv = StateSpace._names(params, prefix), inner + 2 * groups * states
        return [TensorSpec(n["in"], (inner + conv + heads, h)), TensorSpec(n["conv"], (conv, taps)),
                TensorSpec(n["conv_bias"], (conv,)), TensorSpec(n["dt_bias"], (heads,)), TensorSpec(n["A_log"], (heads,)),
                TensorSpec(n["D"], (heads,)), TensorSpec(n["norm"], (inner,), kind="norm"), TensorSpec(n["o"], (h, inner))]

    @staticmethod
    def _ring(params) -> int:
        """Words of a slot's state that the ring takes (padded so that the recurrence's state behind it stays aligned)."""
        heads, size, states, groups, _, taps = StateSpace._sizes(params)
        return (taps * (heads * size + 2 * groups * states) + 3) // 4 * 4 if taps > 1 else 0

    @staticmethod
    def state_request(params):
        heads, size, states, _, _, _ = StateSpace._sizes(params)
        return StateRequest(((StateSpace._ring(params) + heads * states * size + 3) // 4 * 4,), torch.float32)

    def __init__(self, params, tensors, prefix, runtime):
        super().__init__(params, tensors, prefix, runtime)
        self.check_params(params)
        self.hidden, self.eps = int(params["hidden"]), float(params["norm_eps"])
        self.heads, self.size, self.states, self.groups, self.norm_groups, self.taps = self._sizes(params)
        self.inner = self.heads * self.size
        self.conv_width = self.inner + 2 * self.groups * self.states
        n = self._names(params, prefix)
        f32 = lambda t: t.to(torch.float32).contiguous()
        w_in = tensors[n["in"]]
        used = w_in.shape[0]
        self.width = (used + 7) // 8 * 8
        if self.width > used:
            w_in = torch.cat([w_in, torch.zeros((self.width - used, self.hidden), dtype=w_in.dtype, device=w_in.device)])
        self.w_in = prepare_weight(w_in, runtime)
        self.w_o = prepare_weight(tensors[n["o"]], runtime)
        self.conv, self.conv_bias = f32(tensors[n["conv"]].t()), f32(tensors[n["conv_bias"]])
        self.dt_bias, self.skip, self.norm = f32(tensors[n["dt_bias"]]), f32(tensors[n["D"]]), f32(tensors[n["norm"]])
        # bfloat16 with sizes that the tensor-core kernels take: x, B and C are bfloat16 behind the convolution
        self.tensor_cores = runtime.compute_dtype == torch.bfloat16 and ops.ssd_tc_accepts(self.states, self.size)
        self.rate = torch.exp(tensors[n["A_log"]].to(torch.float32)).contiguous()

    def forward(self, ctx, x, residual, scale, kv=None, state=None, store=False, projected=None):
        rt, n = self.runtime, x.shape[0]
        heads, size, states, groups, inner, taps = self.heads, self.size, self.states, self.groups, self.inner, self.taps
        flag, conv = ctx.error_flag, self.conv_width
        slots, split = state.shape[0], self._ring(self.params)
        ring = state[:, :taps * conv].view(slots, taps, conv) if taps > 1 else None
        memory = state[:, split:split + heads * states * size].view(slots, heads, states, size)
        rows = projected
        if rows is None:
            rows = ctx.buffer("ssd.in", (n, self.width), torch.float32)
            linear(rt, STORE, x, self.w_in, rows, error_flag=flag, name="ssd_in")
        z, raw, dt = rows[:, :inner], rows[:, inner:inner + conv], rows[:, inner + conv:inner + conv + heads]
        portions, single = ctx.n_prefill_segments, ctx.decode_rows
        y = ctx.buffer("ssd.y", (n, inner), torch.float32)
        shared = (dt, self.dt_bias, self.rate, self.skip, memory)
        sizes = (heads, groups, states, size)
        if not portions:
            # single tokens alone: the recurrence's kernel does its head's convolution, and its ring, itself
            ops.ssd_single(*shared, single, ctx.slots, y, *sizes,
                           conv=(raw, self.conv, self.conv_bias, ring, ctx.positions, self.tensor_cores))
        else:
            xbc = ctx.buffer("ssd.xbc", (n, conv), torch.bfloat16 if self.tensor_cores else torch.float32)
            ops.ring_conv(raw, None, self.conv, self.conv_bias, ring, ctx.positions, ctx.slots, xbc, act=1)
            if taps > 1:
                ops.ring_store(raw, None, ring, ctx.positions, ctx.slots)
            chunks = ops.ssd_chunks(n - ctx.n_single, portions, self.tensor_cores)
            scratch = ctx.runtime.scratch("ssd.chunks", ops.ssd_scratch_floats(chunks, heads, states, size), torch.float32)
            ops.ssd(xbc, *shared, ctx.prefill_segments, portions, chunks, ctx.slots, y, *sizes, scratch)
            if single.numel():
                ops.ssd_single(*shared, single, ctx.slots, y, *sizes, xbc=xbc)
        o = ctx.buffer("ssd.o", (n, inner), rt.compute_dtype)
        ops.gated_group_norm(y, z, self.norm, ctx.slots, o, self.norm_groups, self.eps)
        linear(rt, STORE if store else ACCUM, o, self.w_o, residual, scale, error_flag=flag, name="ssd_o")
