"""minGRU as a mixer with per-request state.

`mingru`: a gated recurrence per channel whose gates read only the current token.  With z = sigmoid(W_z h + b_z),
u = W_x h + b_x and the candidate c = u + 1/2 where u >= 0, sigmoid(u) where u < 0:

    S_t = (1 - z_t) S_{t-1} + z_t c_t           S_0 = 0
    out_t = W_o (S_t * silu(W_g h_t))

The three projections are ONE product with a 32-bit result; gates, candidate, state and the gated read-out are
32-bit in every engine dtype (csrc/mingru.cu).  The state, `width` floats, is one row per request slot in the
cache manager's state rows: zeroed when a slot is handed out, carried from step to step, so prompt portions of
any length and single decoded tokens continue one another.
"""

from __future__ import annotations

import torch

from ..csrc import kernels
from .base import Mixer, ParamDecl, StateNeed
from .linear import linear
from .registry import register_mixer
from .window_attention import _ProjectsOutput


@register_mixer("mingru")
class MinGRU(Mixer, _ProjectsOutput):
    def __init__(self, hidden_size: int, width: int, names: dict | None = None):
        super().__init__()
        if hidden_size <= 0 or width <= 0:
            raise ValueError("sizes must be positive")
        self.hidden_size, self.width = hidden_size, width
        n = dict(z="z_proj.weight", z_bias="z_proj.bias", x="x_proj.weight", x_bias="x_proj.bias", g="g_proj.weight",
                 o="o_proj.weight")
        n.update(names or {})
        self.names = n

    def param_decls(self):
        H, W, n = self.hidden_size, self.width, self.names
        return {n["z"]: ParamDecl((W, H)), n["z_bias"]: ParamDecl((W,), "bias32"), n["x"]: ParamDecl((W, H)),
                n["x_bias"]: ParamDecl((W,), "bias32"), n["g"]: ParamDecl((W, H)), n["o"]: ParamDecl((H, W))}

    def materialize(self, make):
        H, W, n = self.hidden_size, self.width, self.names
        # one product for the gate's, the candidate's and the output gate's projections
        self.w_in = make("in_proj.weight", ParamDecl((3 * W, H)))
        self.tensors[n["z"]] = self.w_in[:W]
        self.tensors[n["x"]] = self.w_in[W:2 * W]
        self.tensors[n["g"]] = self.w_in[2 * W:]
        self.tensors[n["z_bias"]] = make(n["z_bias"], ParamDecl((W,), "bias32"))
        self.tensors[n["x_bias"]] = make(n["x_bias"], ParamDecl((W,), "bias32"))
        self.tensors[n["o"]] = self._make_o(make, n["o"], (H, W))

    def state_need(self):
        return StateNeed((self.width,), torch.float32)

    def activation_elems(self):
        # the 32-bit product (two elements' worth each in a 16-bit engine), the chunks' scratch, the read-out, the output
        return 6 * self.width + self.width + self.width + self.hidden_size

    def output_projection(self):
        return self.tensors[self.names["o"]], None

    def output_width(self) -> int:
        return self.width

    def forward(self, x, ctx, cache, project_output: bool = True, out=None, out_scale: float = 1.0):
        K = kernels()
        T, W, n, ws = x.shape[0], self.width, self.names, ctx.workspace
        if cache.state is None:
            raise RuntimeError("the minGRU mixer was given no state rows")
        azg = ws.tokens("mingru.in", T, 3 * W, torch.float32)
        K.linear_f32_out(x, self.w_in, azg)
        gated = out if out is not None else ws.tokens("mingru.gated", T, W, x.dtype)
        fold = None
        if ctx.max_q_len > K.mingru_chunk():
            # (a row per token is more than the chunks' pairs ever need: two floats per chunk and channel)
            fold = ws.tokens("mingru.fold", T, W, torch.float32)
        K.mingru(azg, 0, W, 2 * W, self.tensors[n["z_bias"]], self.tensors[n["x_bias"]], cache.state, ctx.cu_q,
                 ctx.req_slots, ctx.token_req, gated, out_scale, ctx.num_requests, ctx.max_q_len, fold)
        if not project_output:
            return gated
        res = ws.tokens("mixer.out", T, self.hidden_size, x.dtype)
        linear(gated, self.tensors[n["o"]], res)
        return res
