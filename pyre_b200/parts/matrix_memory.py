"""A matrix memory with exponential gates (the mLSTM form of xLSTM): a recurrent mixer whose memory is a matrix, a normaliser
and a running maximum per request and head, kept in a state slot of the cache manager."""

from __future__ import annotations

import torch

from ..kernels import lib, ops
from ..weights.specs import TensorSpec
from .base import StateSpec, register_part
from .stacked import StackedMixer, stack_rows


class MatrixMemory(StackedMixer):
    """Per token, with h the mixer's input, ``n_heads`` heads of ``head_dim`` (q, k) and ``v_head_dim`` (v) entries:

        q = W_q h / sqrt(head_dim);  k = W_k h;  v = W_v h
        i = cap tanh((W_i h + b_i) / cap);   f = logsigmoid(cap tanh((W_f h + b_f) / cap))        per head, cap = ``gate_cap``
        m_t = max(f + m_(t-1), i)                                                                 m starts at 0
        S_t = exp(f + m_(t-1) - m_t) S_(t-1) + exp(i - m_t) k_t v_t^T;     n_t likewise with k_t alone
        o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)
        out = W_o [ (o / rms(o) per head) * norm * sigmoid(W_g h) ]                                norm [n_heads * v_head_dim]

    S, n and m live in fp32 in the request's state slot.  The product [q | k | v | g] runs in the compute dtype; the gates'
    logits leave theirs in fp32, and everything from them on, the recurrence, the unit norm and the output gate's product
    are fp32.

    ``names``: the checkpoint's local names."""

    DEFAULT_NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "norm": "norm", "i": "i", "i_bias": "i.b", "f": "f", "f_bias": "f.b"}

    graph_safe = True

    def __init__(self, dtype, device, width: int, n_heads: int, head_dim: int, v_head_dim: int, gate_cap: float, eps: float,
                 names: "dict[str, str] | None" = None):
        super().__init__(dtype, device)
        self.names = dict(self.DEFAULT_NAMES, **(names or {}))
        self.width, self.n_heads, self.head_dim, self.v_head_dim = int(width), int(n_heads), int(head_dim), int(v_head_dim)
        self.gate_cap, self.eps = float(gate_cap), float(eps)
        if min(self.width, self.n_heads, self.head_dim, self.v_head_dim) <= 0 or not self.gate_cap > 0:
            raise ValueError("the sizes and gate_cap of a matrix memory are positive")
        if self.head_dim > ops.STATE_MAX_DIM:
            raise ops.UnsupportedSize(f"heads of {head_dim}: the recurrence takes up to {ops.STATE_MAX_DIM}")
        qk, self.heads_width = self.n_heads * self.head_dim, self.n_heads * self.v_head_dim
        self.k_col, self.v_col, self.g_col = qk, 2 * qk, 2 * qk + self.heads_width
        self.w_gates = self.b_gates = self.norm_w = None

    def tensors(self):
        n, qk, vv, H, W = self.names, self.n_heads * self.head_dim, self.heads_width, self.n_heads, self.width
        return {n["q"]: TensorSpec((qk, W)), n["k"]: TensorSpec((qk, W)), n["v"]: TensorSpec((vv, W)), n["g"]: TensorSpec((vv, W)),
                n["o"]: TensorSpec((W, vv)), n["norm"]: TensorSpec((vv,), role="vector", init=("normal", 1.0, 0.1)),
                n["i"]: TensorSpec((H, W)), n["i_bias"]: TensorSpec((H,), role="vector", init=("normal", -1.0, 1.0)),
                n["f"]: TensorSpec((H, W)), n["f_bias"]: TensorSpec((H,), role="vector", init=("normal", 3.0, 1.0))}

    def load(self, tensors):
        n = self.names
        self.w_in = stack_rows([tensors[n[s]] for s in ("q", "k", "v", "g")])
        self.w_o, self.norm_w = tensors[n["o"]], tensors[n["norm"]]
        self.w_gates = torch.cat([tensors[n["i"]], tensors[n["f"]]], dim=0).contiguous()
        self.b_gates = torch.cat([tensors[n["i_bias"]], tensors[n["f_bias"]]]).contiguous()

    def kernel_libraries(self):
        return ["matrix_state", "elementwise", "gemm_f32" if self.dtype == torch.float32 else "gemm_tc"]

    def cache_spec(self):
        return None

    def state_spec(self):
        return StateSpec((ops.memory_state_floats(self.n_heads, self.head_dim, self.v_head_dim),), torch.float32)

    def head_rows(self, ctx, h, proj, col, call, out=None, out_col=0, scale=1.0):
        st = ctx.state_group(call.state_group)
        with lib.section("gates"):
            gates = ops.linear(h, self.w_gates, out_dtype=torch.float32, partials_ok=True)
        with lib.section("matrix_memory"):
            o, den = ops.matrix_memory(proj, col, col + self.k_col, col + self.v_col, self.head_dim ** -0.5, gates, self.b_gates,
                                       self.gate_cap, st.buffer[call.state_layer], st.slots, ctx.cu_seqlens, self.n_heads, self.head_dim,
                                       self.v_head_dim, lens=ctx.entry_lengths)
        return ops.heads_finish(o, den, self.norm_w, self.eps, proj, col + self.g_col, self.n_heads, self.v_head_dim, self.dtype,
                                gate="sigmoid", post=scale, out=out, out_col=out_col)


register_part("mixer", "matrix_memory", MatrixMemory)
