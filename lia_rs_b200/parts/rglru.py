"""A gated linear recurrent unit behind a short convolution (the recurrent block of Griffin).

    y = gelu(W_y x + b_y),   u = conv(W_x x + b_x)                                     (`width` channels each)
    conv(v)_t[c] = b[c] + sum_j w[c, j] v_(t - taps + 1 + j)[c], zeros before the sequence's start
    r = sigmoid(R_b u_b + br_b),  i = sigmoid(I_b u_b + bi_b)       for each of `blocks` equal parts of the channels
    log a = -8 r softplus(lam);   S_t = a S_(t-1) + sqrt(1 - a^2) i u,   S before the first token = 0 (the first token too)
    out = W_o (S * y)

What a request carries from token to token is one 32-bit state per slot: the convolution's last inputs in a ring of `taps`
rows (csrc/conv_ring.cuh) and S.  The two branches are one product with 32-bit rows.  The convolution's sums and GELU are
32-bit; u is rounded once to the compute element type, and everything behind it (the gates with their products, decays, the
inflow, the state) is 32-bit.  In bfloat16 a step of single tokens is one kernel between the two products
(csrc/rglru_single.cu) and the gates of other steps are a tcgen05 kernel (csrc/rglru_gates_tc.cu).  A step's portions are walked by many warps at once (csrc/rglru.cu), continuing from the slot's
state, so a portion cut anywhere gives what token-by-token steps give, up to the order of the operations.

Parameters: hidden, width, blocks, taps, and optionally `names`."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights import TensorSpec
from .base import Mixer, StateRequest, register_mixer
from .linear import ACCUM, STORE, linear, prepare_weight


@register_mixer("rglru")
class RGLRU(Mixer):
    graph_safe = True
    takes_deferred_norm = True
    can_store = True
    NAMES = {"y": "y", "y_bias": "y.b", "x": "x", "x_bias": "x.b", "conv": "conv", "conv_bias": "conv.b", "r": "ra",
             "r_bias": "ra.b", "i": "ri", "i_bias": "ri.b", "lam": "lam", "o": "o"}

    def graph_key(self, ctx) -> tuple:
        return ()

    @staticmethod
    def _names(params, prefix):
        return {key: prefix + name for key, name in {**RGLRU.NAMES, **params.get("names", {})}.items()}

    @staticmethod
    def check_params(params):
        width, blocks, taps = (int(params[k]) for k in ("width", "blocks", "taps"))
        if width <= 0 or blocks <= 0 or width % blocks:
            raise ValueError("gated linear recurrent unit: blocks must divide width, both positive")
        if width // blocks > ops.RGLRU_MAX_BLOCK:
            raise ValueError(f"gated linear recurrent unit: a part of {width // blocks} channels; the kernel takes "
                             f"{ops.RGLRU_MAX_BLOCK}")
        if not 1 <= taps <= ops.RING_MAX_TAPS:
            raise ValueError(f"gated linear recurrent unit: {taps} taps; the kernel takes 1..{ops.RING_MAX_TAPS}")

    @staticmethod
    def tensor_specs(params, prefix):
        h, width, blocks, taps = (int(params[k]) for k in ("hidden", "width", "blocks", "taps"))
        n, size = RGLRU._names(params, prefix), width // blocks
        return [TensorSpec(n["y"], (width, h)), TensorSpec(n["y_bias"], (width,)), TensorSpec(n["x"], (width, h)),
                TensorSpec(n["x_bias"], (width,)), TensorSpec(n["conv"], (width, taps)), TensorSpec(n["conv_bias"], (width,)),
                TensorSpec(n["r"], (blocks, size, size)), TensorSpec(n["r_bias"], (blocks, size)),
                TensorSpec(n["i"], (blocks, size, size)), TensorSpec(n["i_bias"], (blocks, size)),
                TensorSpec(n["lam"], (width,)), TensorSpec(n["o"], (h, width))]

    @staticmethod
    def _ring(params) -> int:
        """Words of a slot's state that the ring takes (padded so that the recurrence's state behind it stays aligned)."""
        width, taps = int(params["width"]), int(params["taps"])
        return (taps * width + 3) // 4 * 4 if taps > 1 else 0

    @staticmethod
    def state_request(params):
        return StateRequest(((RGLRU._ring(params) + int(params["width"]) + 3) // 4 * 4,), torch.float32)

    def __init__(self, params, tensors, prefix, runtime):
        super().__init__(params, tensors, prefix, runtime)
        self.check_params(params)
        self.hidden, self.width = int(params["hidden"]), int(params["width"])
        self.blocks, self.taps = int(params["blocks"]), int(params["taps"])
        n = self._names(params, prefix)
        f32 = lambda t: t.to(torch.float32).contiguous()
        # one product for both branches, [W_y; W_x], each padded with zero rows to a multiple of 8 columns
        self.branch = (self.width + 7) // 8 * 8
        pad = torch.zeros((self.branch - self.width, self.hidden), dtype=tensors[n["y"]].dtype, device=tensors[n["y"]].device)
        self.w_in = prepare_weight(torch.cat([tensors[n["y"]], pad, tensors[n["x"]], pad], dim=0), runtime)
        self.w_o = prepare_weight(tensors[n["o"]], runtime)
        self.y_bias, self.x_bias = f32(tensors[n["y_bias"]]), f32(tensors[n["x_bias"]])
        self.conv, self.conv_bias = f32(tensors[n["conv"]].t()), f32(tensors[n["conv_bias"]])
        # bfloat16: the tensor-core kernel's matrices as they are stored; else part b's two side by side, transposed
        # ([in][r's outputs | i's outputs])
        self.tensor_cores = runtime.compute_dtype == torch.bfloat16 and ops.rglru_gates_tc_accepts(self.width, self.blocks)
        self.one_kernel = self.tensor_cores and ops.rglru_single_accepts(self.width, self.blocks)
        if self.tensor_cores:
            self.w_r, self.w_i = prepare_weight(tensors[n["r"]], runtime), prepare_weight(tensors[n["i"]], runtime)
        else:
            self.w_gates = prepare_weight(torch.cat([tensors[n["r"]].transpose(1, 2), tensors[n["i"]].transpose(1, 2)], dim=2), runtime)
        self.gate_bias = f32(torch.stack([tensors[n["r_bias"]].reshape(-1), tensors[n["i_bias"]].reshape(-1)]))
        self.rate = (8.0 * torch.nn.functional.softplus(tensors[n["lam"]].to(torch.float32))).contiguous()

    def forward(self, ctx, x, residual, scale, kv=None, state=None, store=False):
        rt, n = self.runtime, x.shape[0]
        width, taps = self.width, self.taps
        flag = ctx.error_flag
        slots, split = state.shape[0], self._ring(self.params)
        ring = state[:, :taps * width].view(slots, taps, width) if taps > 1 else None
        memory = state[:, split:split + width]
        rows = ctx.buffer("rglru.in", (n, 2 * self.branch), torch.float32)
        linear(rt, STORE, x, self.w_in, rows, error_flag=flag, name="yx")
        y, v = rows[:, :width], rows[:, self.branch:self.branch + width]
        out = ctx.buffer("rglru.out", (n, width), rt.compute_dtype)
        if self.one_kernel and ctx.decode_only:
            ops.rglru_single(y, v, self.y_bias, self.x_bias, self.conv, self.conv_bias, self.w_r, self.w_i, self.gate_bias, self.rate,
                             ring, memory, ctx.positions, ctx.slots, out, self.blocks)
            linear(rt, STORE if store else ACCUM, out, self.w_o, residual, scale, error_flag=flag, name="o")
            return
        u = ctx.buffer("rglru.u", (n, width), rt.compute_dtype)
        ops.ring_conv(v, self.x_bias, self.conv, self.conv_bias, ring, ctx.positions, ctx.slots, u)
        a = ctx.buffer("rglru.a", (n, width), torch.float32)
        inflow = ctx.buffer("rglru.inflow", (n, width), torch.float32)
        if self.tensor_cores:
            ops.rglru_gates_tc(u, self.w_r, self.w_i, self.gate_bias, self.rate, ctx.slots, a, inflow, self.blocks, error_flag=flag)
        else:
            ops.rglru_gates(u, self.w_gates, self.gate_bias, self.rate, ctx.slots, a, inflow, self.blocks)
        ops.rglru_scan(a, inflow, y, v, self.y_bias, self.x_bias, ring, memory, ctx.prefill_segments, ctx.n_prefill_segments,
                       ctx.decode_rows, ctx.positions, ctx.slots, out, taps)
        linear(rt, STORE if store else ACCUM, out, self.w_o, residual, scale, error_flag=flag, name="o")
