"""Linear attention with a decay per key channel that depends on the token: a recurrent mixer whose memory is a matrix of
fixed size per request and head, kept in a state slot of the cache manager."""

from __future__ import annotations

import torch

from ..kernels import lib, ops
from ..weights.specs import TensorSpec
from .base import StateSpec, register_part
from .stacked import StackedMixer, stack_rows


class GatedLinearAttention(StackedMixer):
    """Per token, with h the mixer's input, ``n_heads`` heads of ``head_dim`` (q, k) and ``v_head_dim`` (v) entries:

        q = W_q h / sqrt(head_dim);  k = W_k h;  v = W_v h
        alpha = sigmoid(W_a2 W_a1 h + b)^(1 / tau)                 one decay per head and key channel, ``decay_rank`` inner size
        head n:  S_t = diag(alpha_t) S_(t-1) + k_t v_t^T;   o_t = S_t^T q_t
        out = W_o [ (o / rms(o) per head) * norm * silu(W_g h) ]      norm [v_head_dim], shared by the heads

    S [head_dim, v_head_dim] per head lives in fp32 in the request's state slot.  The product [a1 | q | k | v | g] runs in the
    compute dtype, as does the decay's second map, whose result leaves the product in fp32; the decay from there on, the
    recurrence, the unit norm and the gate's product are fp32.

    ``names``: the checkpoint's local names."""

    DEFAULT_NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "norm": "norm", "a1": "a1", "a2": "a2", "a2_bias": "a2.b"}

    graph_safe = True

    def __init__(self, dtype, device, width: int, n_heads: int, head_dim: int, v_head_dim: int, decay_rank: int, tau: float, eps: float,
                 names: "dict[str, str] | None" = None):
        super().__init__(dtype, device)
        self.names = dict(self.DEFAULT_NAMES, **(names or {}))
        self.width, self.n_heads, self.head_dim, self.v_head_dim = int(width), int(n_heads), int(head_dim), int(v_head_dim)
        self.decay_rank, self.tau, self.eps = int(decay_rank), float(tau), float(eps)
        if min(self.width, self.n_heads, self.head_dim, self.v_head_dim, self.decay_rank) <= 0 or not self.tau > 0:
            raise ValueError("the sizes and tau of a gated linear attention are positive")
        if self.head_dim > ops.STATE_MAX_DIM:
            raise ops.UnsupportedSize(f"heads of {head_dim}: the recurrence takes up to {ops.STATE_MAX_DIM}")
        qk, self.heads_width = self.n_heads * self.head_dim, self.n_heads * self.v_head_dim
        # the decay's inner columns come first, padded by zero rows to a multiple of 8: both products of the decay then have
        # operands on 16-byte boundaries
        self.inner = -(-self.decay_rank // 8) * 8
        self.q_col, self.k_col, self.v_col = self.inner, self.inner + qk, self.inner + 2 * qk
        self.g_col = self.v_col + self.heads_width
        self.w_a2 = self.b_a2 = self.norm_w = None

    def tensors(self):
        n, qk, vv = self.names, self.n_heads * self.head_dim, self.heads_width
        return {n["q"]: TensorSpec((qk, self.width)), n["k"]: TensorSpec((qk, self.width)), n["v"]: TensorSpec((vv, self.width)),
                n["g"]: TensorSpec((vv, self.width)), n["o"]: TensorSpec((self.width, vv)),
                n["norm"]: TensorSpec((self.v_head_dim,), role="vector", init=("normal", 1.0, 0.1)),
                n["a1"]: TensorSpec((self.decay_rank, self.width)),
                n["a2"]: TensorSpec((qk, self.decay_rank), init=("normal", 0.0, 0.3)),
                n["a2_bias"]: TensorSpec((qk,), role="vector", init=("normal", 1.0, 1.0))}

    def load(self, tensors):
        n = self.names
        pad = self.inner - self.decay_rank
        a1 = torch.nn.functional.pad(tensors[n["a1"]], (0, 0, 0, pad))
        self.w_in = stack_rows([a1] + [tensors[n[s]] for s in ("q", "k", "v", "g")])
        self.w_o, self.norm_w = tensors[n["o"]], tensors[n["norm"]]
        self.w_a2, self.b_a2 = torch.nn.functional.pad(tensors[n["a2"]], (0, pad)).contiguous(), tensors[n["a2_bias"]]

    def kernel_libraries(self):
        return ["matrix_state", "elementwise", "gemm_f32" if self.dtype == torch.float32 else "gemm_tc"]

    def cache_spec(self):
        return None

    def state_spec(self):
        return StateSpec((self.n_heads * self.head_dim * self.v_head_dim,), torch.float32)

    def head_rows(self, ctx, h, proj, col, call, out=None, out_col=0, scale=1.0):
        st = ctx.state_group(call.state_group)
        with lib.section("decay"):
            z = ops.linear(proj[:, col:col + self.inner], self.w_a2, out_dtype=torch.float32)
        o = ops.gated_linear_attention(proj, col + self.q_col, col + self.k_col, col + self.v_col, self.head_dim ** -0.5, z, self.b_a2, self.tau,
                                       st.buffer[call.state_layer], st.slots, ctx.cu_seqlens, self.n_heads, self.head_dim, self.v_head_dim,
                                       lens=ctx.entry_lengths)
        return ops.heads_finish(o, None, self.norm_w, self.eps, proj, col + self.g_col, self.n_heads, self.v_head_dim, self.dtype,
                                gate="silu", post=scale, out=out, out_col=out_col)


register_part("mixer", "gated_linear_attention", GatedLinearAttention)
