"""Linear attention with one fixed decay per head and per-request state.

    q = silu(W_q h), k = silu(W_k h) (heads x dim), v = silu(W_v h) (heads x value_dim)
    S_t = decay_h S_{t-1} + k_t v_t^T        S [dim, value_dim], S_0 = 0
    o_t = S_t^T q_t
    out = W_o (norm_w * n(o) * sigmoid(W_g h))        n: the concatenated heads by their common root mean square

It is the state-space recurrence of csrc/ssd.cu and csrc/ssd_chunk.cu with x = v, B = k, C = q (a group per head), steps of
one and decays that do not depend on the token, so it runs on those kernels: prompt portions in chunks on the tensor cores
where the sizes allow, everything else token by token.  State, decays, read-out and norm are 32-bit in every engine dtype.
The state row of a request holds S of every head; it is zeroed when a slot is handed out and carried from step to step.
"""

from __future__ import annotations

import math

import torch

from ..csrc import kernels
from .base import Mixer, ParamDecl, StateNeed
from .linear import linear
from .mamba2 import CHUNK_LEAST
from .registry import register_mixer


@register_mixer("fixed_decay_attention")
class FixedDecayAttention(Mixer):
    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, value_dim: int, decay, eps: float,
                 names: dict | None = None):
        """`decay`: one number in (0, 1] per head.  `names`: the checkpoint's names of q, k, v, gate, o, norm behind the
        mixer's prefix."""
        super().__init__()
        if min(hidden_size, num_heads, head_dim, value_dim) <= 0:
            raise ValueError("sizes must be positive")
        if head_dim > 512:
            raise ValueError(f"head_dim={head_dim}: the recurrence kernel takes up to 512")
        self.decay = [float(d) for d in decay]
        if len(self.decay) != num_heads or not all(0.0 < d <= 1.0 for d in self.decay):
            raise ValueError(f"decay={decay}: one number above 0 and at most 1 for each of {num_heads} heads")
        self.hidden_size, self.num_heads, self.head_dim, self.value_dim, self.eps = hidden_size, num_heads, head_dim, value_dim, float(eps)
        n = dict(q="q_proj.weight", k="k_proj.weight", v="v_proj.weight", gate="g_proj.weight", o="o_proj.weight",
                 norm="norm.weight")
        n.update(names or {})
        self.names = n
        self.qk_size, self.v_size = num_heads * head_dim, num_heads * value_dim

    def param_decls(self):
        H, n = self.hidden_size, self.names
        return {n["q"]: ParamDecl((self.qk_size, H)), n["k"]: ParamDecl((self.qk_size, H)), n["v"]: ParamDecl((self.v_size, H)),
                n["gate"]: ParamDecl((self.v_size, H)), n["o"]: ParamDecl((H, self.v_size)),
                n["norm"]: ParamDecl((self.v_size,), "norm")}

    def materialize(self, make):
        H, n, qk, vs = self.hidden_size, self.names, self.qk_size, self.v_size
        # one product with rows v | k | q | gate: the recurrence's x, B and C in its kernels' order, the gate behind
        self.w_in = make("in_proj.weight", ParamDecl((2 * qk + 2 * vs, H)))
        self.tensors[n["v"]] = self.w_in[:vs]
        self.tensors[n["k"]] = self.w_in[vs:vs + qk]
        self.tensors[n["q"]] = self.w_in[vs + qk:vs + 2 * qk]
        self.tensors[n["gate"]] = self.w_in[vs + 2 * qk:]
        self.tensors[n["o"]] = make(n["o"], ParamDecl((H, vs)))
        self.tensors[n["norm"]] = make(n["norm"], ParamDecl((vs,), "norm"))

    def weights_loaded(self):
        dev = self.w_in.device
        # the recurrence's steps, logarithms of decays (one row that serves all tokens) and skip weights
        self.steps = torch.ones(1, self.num_heads, dtype=torch.float32, device=dev)
        self.log_decay = torch.tensor([[math.log(d) for d in self.decay]], dtype=torch.float32, device=dev)
        self.skip = torch.zeros(self.num_heads, dtype=torch.float32, device=dev)

    def state_need(self):
        return StateNeed((self.num_heads * self.value_dim * self.head_dim,), torch.float32)

    def activation_elems(self):
        # the input product, o in 32-bit (two elements' worth), the gated o, the output, the chunked form's scores
        return 2 * self.qk_size + 5 * self.v_size + self.hidden_size + 128 * self.num_heads

    def operand_dtype(self):
        return self.w_in.dtype

    def output_projection(self):
        return self.tensors[self.names["o"]], None

    def forward(self, x, ctx, cache, project_output: bool = True):
        K, T, n, t, ws = kernels(), x.shape[0], self.names, self.tensors, ctx.workspace
        N, d, dv, qk, vs = self.num_heads, self.head_dim, self.value_dim, self.qk_size, self.v_size
        if cache.state is None:
            raise RuntimeError("the linear attention mixer was given no state rows")
        u = ws.tokens("lin.in", T, 2 * qk + 2 * vs, x.dtype)
        linear(x, self.w_in, u)
        o = ws.tokens("lin.o", T, vs, torch.float32)
        chunked = ctx.max_q_len > CHUNK_LEAST and K.ssd_chunk_applies(x.dtype, N, d, dv, N)
        if chunked:
            K.act_rows("silu", u[:, :vs + 2 * qk], u[:, :vs + 2 * qk])
            scores = ws.tokens("ssd.scores", T, K.ssd_chunk_floats(1, N), torch.float32)
            K.ssd_chunk(u, vs, vs + qk, self.steps, self.log_decay, self.skip, scores, cache.state, ctx.cu_q, ctx.req_slots,
                        ctx.token_req, o, ctx.num_requests, N, d, dv, N, CHUNK_LEAST)
        if not chunked or ctx.num_requests > 1:
            K.ssd_recurrence(u, vs, vs + qk, self.steps, self.log_decay, self.skip, cache.state, ctx.cu_q, ctx.req_slots,
                             ctx.token_req, o, ctx.num_requests, N, d, dv, N, CHUNK_LEAST if chunked else 1 << 30,
                             silu_in=not chunked, single=ctx.max_q_len == 1)
        g = ws.tokens("lin.gated", T, vs, x.dtype)
        K.ssd_gate_norm(o, u[:, vs + 2 * qk:], t[n["norm"]], 1, self.eps, g, gate_behind=True)
        if not project_output:
            return g
        out = ws.tokens("mixer.out", T, self.hidden_size, x.dtype)
        linear(g, t[n["o"]], out)
        return out
