"""A state-space mixer with a scalar decay per head (Mamba-2, "state-space duality") and per-request state.

With inner = heads * value_dim, N = `state`, G = `groups` and W_in h laid out as [z: inner | x: inner | B: G N | C: G N |
dt: heads]:

    x | B | C  <-  silu(causal convolution over time, per channel, with a bias)
    dt = softplus(dt + dt_bias);   head h reads B and C of group h / (heads / G)
    S_t = exp(-exp(A_log) dt_t) S_{t-1} + dt_t B_t x_t^T         S [N, value_dim], S_0 = 0
    y_t = S_t^T C_t + D x_t
    out = W_o (norm_w * n(y * silu(z)))        n: every one of `norm_groups` equal parts by its own root mean square

The convolved rows are the engine's dtype; steps, decays, state, read-out and norm are 32-bit in every engine dtype
(csrc/ssd.cu).  The state row of a request holds S of every head and the convolution's last taps - 1 projected rows; it is
zeroed when a slot is handed out and carried from step to step, over any mix of prompt portions and single tokens.
"""

from __future__ import annotations

import torch

from ..csrc import kernels
from .base import Mixer, ParamDecl, SharesInput, StateNeed
from .linear import linear
from .registry import register_mixer


CHUNK_LEAST = 16  # requests that bring more tokens than this take the chunked form


def _up4(n: int) -> int:
    return -(-n // 4) * 4


@register_mixer("mamba2")
class Mamba2(Mixer, SharesInput):
    def __init__(self, hidden_size: int, num_heads: int, value_dim: int, state: int, groups: int, conv_taps: int,
                 norm_groups: int, eps: float, names: dict | None = None):
        """`names`: the checkpoint's names of in, conv, conv_bias, dt_bias, a_log, d, norm, o behind the mixer's prefix."""
        super().__init__()
        if min(hidden_size, num_heads, value_dim, state, groups, norm_groups) <= 0:
            raise ValueError("sizes must be positive")
        if num_heads % groups or (num_heads * value_dim) % norm_groups:
            raise ValueError("num_heads must be a multiple of groups and the inner size one of norm_groups")
        if state > 512 or not 1 <= conv_taps <= 32:
            raise ValueError(f"state={state}, conv_taps={conv_taps}: the kernels take up to 512 and 1 to 32 taps")
        self.hidden_size, self.num_heads, self.value_dim, self.state, self.groups = hidden_size, num_heads, value_dim, state, groups
        self.conv_taps, self.norm_groups, self.eps = conv_taps, norm_groups, float(eps)
        n = dict(in_proj="in_proj.weight", conv="conv1d.weight", conv_bias="conv1d.bias", dt_bias="dt_bias", a_log="A_log",
                 d="D", norm="norm.weight", o="out_proj.weight")
        n.update(names or {})
        self.names = n
        self.inner = num_heads * value_dim
        self.channels = self.inner + 2 * groups * state  # x | B | C
        self.s_floats = _up4(num_heads * value_dim * state)
        self.conv_floats = _up4((conv_taps - 1) * self.channels)

    def input_width(self):
        return self.inner + self.channels + self.num_heads

    def param_decls(self):
        H, n = self.hidden_size, self.names
        return {
            n["in_proj"]: ParamDecl((self.input_width(), H)), n["conv"]: ParamDecl((self.channels, self.conv_taps)),
            n["conv_bias"]: ParamDecl((self.channels,), "bias32"), n["dt_bias"]: ParamDecl((self.num_heads,), "bias32"),
            n["a_log"]: ParamDecl((self.num_heads,), "bias32"), n["d"]: ParamDecl((self.num_heads,), "norm"),
            n["norm"]: ParamDecl((self.inner,), "norm"), n["o"]: ParamDecl((H, self.inner)),
        }

    def materialize(self, make):
        n = self.names
        for name, decl in self.param_decls().items():
            self.tensors[name] = self._make_in(make, name, decl.shape) if name == n["in_proj"] else make(name, decl)

    def state_need(self):
        return StateNeed((self.s_floats + self.conv_floats,), torch.float32)

    def activation_elems(self):
        # the input product, the convolved rows, steps and decays and y in 32-bit (two elements each), the gated y, the output
        # ... and the chunked form's scores
        return (self.input_width() + self.channels + 4 * self.num_heads + 3 * self.inner + self.hidden_size
                + 128 * self.groups)

    def output_projection(self):
        return self.tensors[self.names["o"]], None

    def forward(self, x, ctx, cache, project_output: bool = True, projected=None, out=None):
        K = kernels()
        T, n, t, ws = x.shape[0], self.names, self.tensors, ctx.workspace
        N, P, S, G, inner, ch = self.num_heads, self.value_dim, self.state, self.groups, self.inner, self.channels
        if cache.state is None:
            raise RuntimeError("the state-space mixer was given no state rows")
        u = projected
        if u is None:
            u = ws.tokens("ssd.in", T, self.input_width(), x.dtype)
            linear(x, t[n["in_proj"]], u)
        conv_state = cache.state[:, self.s_floats:]
        xbc = ws.tokens("ssd.xbc", T, ch, x.dtype)
        dt = ws.tokens("ssd.dt", T, N, torch.float32)
        log_decay = ws.tokens("ssd.log_decay", T, N, torch.float32)
        K.ssd_prepare(u, inner, inner + ch, t[n["conv"]], t[n["conv_bias"]], t[n["dt_bias"]], t[n["a_log"]], conv_state,
                      ctx.cu_q, ctx.token_req, ctx.req_slots, xbc, dt, log_decay, single=ctx.max_q_len == 1)
        if self.conv_taps > 1 and ctx.max_q_len > 1:
            K.conv_state_update(u[:, inner:inner + ch], self.conv_taps, conv_state, ctx.cu_q, ctx.token_req, ctx.req_slots,
                                ctx.num_requests)
        y = ws.tokens("ssd.y", T, inner, torch.float32)
        # prompt portions in chunks on the tensor cores (16-bit, at the sizes that form takes), the rest token by token
        chunked = ctx.max_q_len > CHUNK_LEAST and K.ssd_chunk_applies(x.dtype, N, S, P, G)
        if chunked:
            scores = ws.tokens("ssd.scores", T, K.ssd_chunk_floats(1, G), torch.float32)
            K.ssd_chunk(xbc, inner, inner + G * S, dt, log_decay, t[n["d"]], scores, cache.state, ctx.cu_q, ctx.req_slots,
                        ctx.token_req, y, ctx.num_requests, N, S, P, G, CHUNK_LEAST)
        if not chunked or ctx.num_requests > 1:
            K.ssd_recurrence(xbc, inner, inner + G * S, dt, log_decay, t[n["d"]], cache.state, ctx.cu_q, ctx.req_slots,
                             ctx.token_req, y, ctx.num_requests, N, S, P, G, CHUNK_LEAST if chunked else 1 << 30,
                             single=ctx.max_q_len == 1)
        g = ws.tokens("ssd.gated", T, inner, x.dtype)
        K.ssd_gate_norm(y, u[:, :inner], t[n["norm"]], self.norm_groups, self.eps, g)
        if not project_output:
            return g
        if out is None:
            out = ws.tokens("mixer.out", T, self.hidden_size, x.dtype)
        linear(g, t[n["o"]], out)
        return out
