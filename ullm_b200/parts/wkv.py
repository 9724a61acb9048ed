"""Time mixing with a decay per key channel and a bonus for the current token (RWKV-style), with per-request state.

With h' the row before h (zeros in front of the first), each of r, k, v, g, w reads its own mix h + (h' - h) * mu_s:

    r, k, v = W_r, W_k, W_v of their mixes (heads x dim);   gate = silu(W_g of its mix)
    w = exp(-exp(W_w2 tanh(W_w1 of its mix) + w0))          a decay per head and key channel
    o_t = (S_{t-1} + diag(u) k_t v_t^T)^T r_t               u: the bonus, per head and key channel
    S_t = diag(w_t) S_{t-1} + k_t v_t^T                     S [dim, dim], S_0 = 0
    out = W_o (norm_w * n(o) * gate)                        n: each head by its own root mean square

The five mixes are one kernel, the five products (r | k | v | g | w1, stacked; an operand each) one launch in decode steps and
a batched product in prompts, the low-rank decay one kernel (csrc/token_shift.cu); the recurrence is that of csrc/gla.cu
and csrc/gla_chunk.cu with their bonus.  Decays, state, read-out and norms are 32-bit in every engine dtype.  The state row of a request holds S of
every head and the last row h; it is zeroed when a slot is handed out and carried from step to step.
"""

from __future__ import annotations

import torch

from ..csrc import kernels
from .base import Mixer, ParamDecl, StateNeed
from .linear import linear
from .mamba2 import CHUNK_LEAST
from .registry import register_mixer

_MIXES = ("r", "k", "v", "g", "w")


def _up(n: int, m: int) -> int:
    return -(-n // m) * m


@register_mixer("wkv")
class TimeMixing(Mixer):
    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, decay_rank: int, eps: float,
                 names: dict | None = None):
        """`decay_rank`: the inner size of the decay's projection.  `names`: the checkpoint's names of mu (a format string
        taking r, k, v, g or w), r, k, v, g, w1, w2, w0, u, norm, o behind the mixer's prefix."""
        super().__init__()
        if min(hidden_size, num_heads, head_dim, decay_rank) <= 0:
            raise ValueError("sizes must be positive")
        if head_dim > 512:
            raise ValueError(f"head_dim={head_dim}: the recurrence kernel takes up to 512")
        self.hidden_size, self.num_heads, self.head_dim, self.decay_rank, self.eps = hidden_size, num_heads, head_dim, decay_rank, float(eps)
        n = dict(mu="mu_{}", r="r_proj.weight", k="k_proj.weight", v="v_proj.weight", g="g_proj.weight", w1="w_proj.0.weight",
                 w2="w_proj.1.weight", w0="w_proj.1.bias", u="bonus", norm="norm.weight", o="o_proj.weight")
        n.update(names or {})
        self.names = n
        self.size = num_heads * head_dim
        self.rank_rows = _up(decay_rank, 8)  # (rows of zeros fill the decay's part: the product's rows stay on 16-byte borders)
        self.s_floats = _up(num_heads * head_dim * head_dim, 4)

    def _decls(self):
        H, n, S, R = self.hidden_size, self.names, self.size, self.decay_rank
        d = {n["mu"].format(s): ParamDecl((H,), "bias32") for s in _MIXES}
        d.update({n[s]: ParamDecl((S, H)) for s in "rkvg"})
        d.update({n["w1"]: ParamDecl((R, H)), n["w2"]: ParamDecl((S, R)), n["w0"]: ParamDecl((S,), "bias32"),
                  n["u"]: ParamDecl((self.num_heads, self.head_dim), "bias32"), n["norm"]: ParamDecl((S,), "norm"),
                  n["o"]: ParamDecl((H, S))})
        return d

    def param_decls(self):
        return self._decls()

    def materialize(self, make):
        H, n, S, R = self.hidden_size, self.names, self.size, self.decay_rank
        # the five products' weights stacked, r | k | v | g | w1, and the five mixing vectors
        self.w_in = make("in_proj.weight", ParamDecl((4 * S + self.rank_rows, H)))
        self.w_in[4 * S + R:].zero_()
        self.mu = make("mu", ParamDecl((5, H), "bias32"))
        for i, s in enumerate(_MIXES):
            self.tensors[n["mu"].format(s)] = self.mu[i]
            if s != "w":
                self.tensors[n[s]] = self.w_in[i * S:(i + 1) * S]
        self.tensors[n["w1"]] = self.w_in[4 * S:4 * S + R]
        for name, decl in self._decls().items():
            if name not in self.tensors:
                self.tensors[name] = make(name, decl)

    def state_need(self):
        return StateNeed((self.s_floats + _up(self.hidden_size, 4),), torch.float32)

    def activation_elems(self):
        # the mixes, the input products, decays and o in 32-bit (two elements each), the gated o, the output
        return 5 * self.hidden_size + 4 * self.size + self.rank_rows + 5 * self.size + self.hidden_size

    def operand_dtype(self):
        return self.w_in.dtype

    def output_projection(self):
        return self.tensors[self.names["o"]], None

    def forward(self, x, ctx, cache, project_output: bool = True):
        K, T, n, t, ws = kernels(), x.shape[0], self.names, self.tensors, ctx.workspace
        H, S, N, d = self.hidden_size, self.size, self.num_heads, self.head_dim
        if cache.state is None:
            raise RuntimeError("the time-mixing mixer was given no state rows")
        mixes = ws.get("wkv.mixes", 5 * T, H, x.dtype, reserve=5 * ws.max_tokens).view(5, T, H)
        K.token_shift_mix(x, self.mu, mixes, cache.state[:, self.s_floats:], ctx.cu_q, ctx.token_req, ctx.req_slots,
                          ctx.num_requests, single=ctx.max_q_len == 1)
        y = ws.tokens("wkv.in", T, 4 * S + self.rank_rows, x.dtype)
        K.grouped_linear(mixes, self.w_in, y, S)
        w = ws.tokens("wkv.decay", T, S, torch.float32)
        K.low_rank_decay(y[:, 4 * S:4 * S + self.decay_rank], t[n["w2"]], t[n["w0"]], w)
        o = ws.tokens("wkv.o", T, S, torch.float32)
        # prompt portions in chunks on the tensor cores (16-bit, at the sizes that form takes), the rest token by token
        chunked = ctx.max_q_len > CHUNK_LEAST and K.gla_chunk_applies(x.dtype, N, d, d)
        if chunked:
            scratch = K.gla_chunk_scratch(ws, T, ctx.num_requests, N, d, d)
            K.gla_chunk(y, 0, S, 2 * S, w, 1.0, scratch, cache.state, ctx.cu_q, ctx.req_slots, ctx.token_req, o,
                        ctx.num_requests, N, d, d, CHUNK_LEAST, bonus=t[n["u"]])
        if not chunked or ctx.num_requests > 1:
            K.gla_recurrence(y, 0, S, 2 * S, w, None, 0.0, 1.0, cache.state, ctx.cu_q, ctx.req_slots, ctx.token_req, o,
                             ctx.num_requests, N, d, d, bonus=t[n["u"]], most_tokens=CHUNK_LEAST if chunked else 1 << 30,
                             single=ctx.max_q_len == 1)
        g = ws.tokens("wkv.gated", T, S, x.dtype)
        K.head_norm_gate(o, y[:, 3 * S:4 * S], t[n["norm"]], self.eps, g, N, d, silu=True)
        if not project_output:
            return g
        out = ws.tokens("mixer.out", T, H, x.dtype)
        linear(g, t[n["o"]], out)
        return out
