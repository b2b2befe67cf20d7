"""A matrix memory with exponential gates (mLSTM, the matrix memory of xLSTM).

    q = W_q x * head_dim^(-1/2), k = W_k x  (heads x head_dim),  v = W_v x, g = W_g x  (heads x v_head_dim)
    log gates, one a head:  i = cap tanh((W_i x + b_i) / cap),  f = log sigmoid(cap tanh((W_f x + b_f) / cap))
    m_t = max(f_t + m_(t-1), i_t)                                 (m, S and n are zero before a request's first token)
    S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t^T,   n_t likewise with k_t alone
    o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)
    out = W_o ( concat_h(o_t,h / sqrt(mean(o_t,h^2) + eps)) * w * sigmoid(g_t) ),   w [heads v_head_dim]

What a request carries from token to token is one 32-bit state per slot: S of all heads, then n, then m.  The six input
products are one product against [W_q; W_k; W_v; W_g; W_i; W_f] with 32-bit output in a step of single tokens; with prompt
portions, where the tensor-core kernels take the sizes (bfloat16), the first three are a product of their own whose rows are
bfloat16, and single tokens always see q, k and v rounded so.  Gates, exponents, the state, every sum over it and the heads'
norm are 32-bit (csrc/mlstm.cu, csrc/mlstm_tc.cu).  Single tokens update the state in place; prompt portions are cut into
chunks that run side by side and continue from the slot's state, so a portion cut anywhere gives what token-by-token steps
give, up to the order of the additions.

Parameters: hidden, heads, head_dim, v_head_dim, gate_cap, norm_eps, and optionally `names`."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights import TensorSpec
from .base import Mixer, StateRequest, register_mixer
from .linear import ACCUM, STORE, linear, prepare_weight


@register_mixer("mlstm")
class MatrixMemory(Mixer):
    graph_safe = True
    takes_deferred_norm = True
    can_store = True
    NAMES = {"q": "q", "k": "k", "v": "v", "gate": "g", "o": "o", "norm": "norm", "i": "i", "i_bias": "i.b", "f": "f",
             "f_bias": "f.b"}

    def graph_key(self, ctx) -> tuple:
        return ()            # the chunks' number follows from the step's numbers of tokens, single tokens and portions

    @staticmethod
    def _names(params, prefix):
        return {key: prefix + name for key, name in {**MatrixMemory.NAMES, **params.get("names", {})}.items()}

    @staticmethod
    def _sizes(params):
        return tuple(int(params[k]) for k in ("heads", "head_dim", "v_head_dim"))

    @staticmethod
    def check_params(params):
        heads, d, dv = MatrixMemory._sizes(params)
        if heads <= 0 or not 0 < d <= ops.MLSTM_MAX_HEAD or not 0 < dv <= ops.MLSTM_MAX_HEAD:
            raise ValueError(f"matrix memory: heads positive, head_dim and v_head_dim within 1..{ops.MLSTM_MAX_HEAD} "
                             "(what the kernel takes)")
        if not float(params["gate_cap"]) > 0:
            raise ValueError("matrix memory: gate_cap must be positive")

    @staticmethod
    def tensor_specs(params, prefix):
        h, (heads, d, dv) = int(params["hidden"]), MatrixMemory._sizes(params)
        n = MatrixMemory._names(params, prefix)
        return [TensorSpec(n["q"], (heads * d, h)), TensorSpec(n["k"], (heads * d, h)), TensorSpec(n["v"], (heads * dv, h)),
                TensorSpec(n["gate"], (heads * dv, h)), TensorSpec(n["i"], (heads, h)), TensorSpec(n["i_bias"], (heads,)),
                TensorSpec(n["f"], (heads, h)), TensorSpec(n["f_bias"], (heads,)),
                TensorSpec(n["norm"], (heads * dv,), kind="norm"), TensorSpec(n["o"], (h, heads * dv))]

    @staticmethod
    def state_request(params):
        heads, d, dv = MatrixMemory._sizes(params)
        return StateRequest(((heads * (d * dv + d + 1) + 3) // 4 * 4,), torch.float32)

    def __init__(self, params, tensors, prefix, runtime):
        super().__init__(params, tensors, prefix, runtime)
        self.check_params(params)
        self.hidden = int(params["hidden"])
        self.heads, self.d, self.dv = self._sizes(params)
        self.eps, self.cap = float(params["norm_eps"]), float(params["gate_cap"])
        n = self._names(params, prefix)
        blocks = [tensors[n[key]] for key in ("q", "k", "v", "gate", "i", "f")]
        self.split = self.heads * (2 * self.d + self.dv)              # q, k and v; behind them what stays 32-bit
        used = sum(block.shape[0] for block in blocks)
        self.width = (used + 7) // 8 * 8
        if self.width > used:
            blocks.append(torch.zeros((self.width - used, self.hidden), dtype=blocks[0].dtype, device=blocks[0].device))
        self.w_in = prepare_weight(torch.cat(blocks, dim=0), runtime)
        self.w_o = prepare_weight(tensors[n["o"]], runtime)
        f32 = lambda t: t.to(torch.float32).contiguous()
        self.i_bias, self.f_bias, self.norm = f32(tensors[n["i_bias"]]), f32(tensors[n["f_bias"]]), f32(tensors[n["norm"]])
        # bfloat16 with sizes that the tensor-core kernels take: q, k and v are bfloat16 behind their product
        self.pieces = ops.mlstm_tc_pieces(self.d, self.dv) if runtime.compute_dtype == torch.bfloat16 else 0

    def forward(self, ctx, x, residual, scale, kv=None, state=None, store=False):
        rt, n, flag = self.runtime, x.shape[0], ctx.error_flag
        heads, d, dv = self.heads, self.d, self.dv
        portions, single = ctx.n_prefill_segments, ctx.decode_rows
        tensor_cores = self.pieces > 0 and portions > 0
        if tensor_cores:
            qkv = ctx.buffer("mlstm.qkv", (n, self.split), rt.compute_dtype)
            gates = ctx.buffer("mlstm.gates", (n, self.width - self.split), torch.float32)
            linear(rt, STORE, x, self.w_in[:self.split], qkv, error_flag=flag, name="mlstm_qkv")
            linear(rt, STORE, x, self.w_in[self.split:], gates, error_flag=flag, name="mlstm_gates")
        else:
            rows = ctx.buffer("mlstm.in", (n, self.width), torch.float32)
            linear(rt, STORE, x, self.w_in, rows, error_flag=flag, name="mlstm_in")
            qkv, gates = rows[:, :self.split], rows[:, self.split:]
        o = ctx.buffer("mlstm.o", (n, heads * dv), rt.compute_dtype)
        shared = (qkv, gates, self.i_bias, self.f_bias, self.cap, state)
        if portions:
            chunks = ops.mlstm_chunks(n - ctx.n_single, portions, tensor_cores)
            scratch = ctx.runtime.scratch("mlstm.chunks", ops.mlstm_scratch_floats(chunks, heads, d, dv), torch.float32)
            y = ctx.buffer("mlstm.y", (n, heads * dv), torch.float32) if tensor_cores and self.pieces > 1 else None
            ops.mlstm(*shared, ctx.prefill_segments, portions, chunks, ctx.slots, self.norm, self.eps, o, heads, d, dv, scratch, y=y)
        if single.numel():
            ops.mlstm_single(*shared, single, ctx.slots, self.norm, self.eps, o, heads, d, dv, round16=self.pieces > 0,
                             wanted_ctas=2 * ctx.runtime.sm_count)
        linear(rt, STORE if store else ACCUM, o, self.w_o, residual, scale, error_flag=flag, name="o")
