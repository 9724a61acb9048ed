"""Two mixers run side by side on the same rows.

`parallel_mixers`: result = left_scale * left(h) + right_scale * right(h) for two mixers that read the same rows.
Both stop in front of their output projections and leave their rows, already scaled, side by side in one buffer;
ONE product with the two projections' weights side by side [hidden, left width + right width] forms the sum.
At most one of the two keeps pages and at most one keeps state rows; each finds them in the execution's cache.

`parallel_normed_mixers`: result = mult * (RMSnorm(left(h)) + RMSnorm(right(h))), each norm over the model width with a
weight of its own.  Both may keep state: their rows lie side by side in the execution's.  The norms stand between the output projections and the sum, so there are two projections; but both
mixers read the same rows, so their input projections are ONE product (rows left | right), of which each gets its
column range.  Norms, sum and the addition to a 32-bit stream are one kernel, which also leaves the rows of the norm
that reads the stream next (`forward_add`).
"""

from __future__ import annotations

from dataclasses import replace

import torch

from ..csrc import kernels
from .base import Mixer, ParamDecl, SharesInput, StateNeed
from .linear import linear
from .registry import build_mixer, register_mixer
from .window_attention import _ProjectsOutput


def _check_caches(left, right):
    if sum(m.cache_need() is not None for m in (left, right)) > 1:
        raise ValueError("at most one of two mixers side by side keeps pages")
    if sum(m.state_need() is not None for m in (left, right)) > 1:
        raise ValueError("at most one of two mixers side by side keeps state rows")


@register_mixer("parallel_mixers")
class ParallelMixers(Mixer):
    def __init__(self, hidden_size: int, left, right, left_scale: float = 1.0, right_scale: float = 1.0,
                 names: dict | None = None):
        """`left`, `right`: `MixerSpec`s of mixers that can stop in front of their output projection
        (`forward(..., project_output=False, out=, out_scale=)`, `output_width()`, a shareable `o` weight).
        `names`: the prefixes of the two mixers' tensors behind this mixer's own prefix."""
        super().__init__()
        self.hidden_size = hidden_size
        self.left, self.right = build_mixer(left), build_mixer(right)
        self.left_scale, self.right_scale = float(left_scale), float(right_scale)
        for m in (self.left, self.right):
            if not isinstance(m, _ProjectsOutput):
                raise ValueError(f"{type(m).__name__} cannot hand its output projection to a caller")
        _check_caches(self.left, self.right)
        n = dict(left="left.", right="right.")
        n.update(names or {})
        self.names = n

    def subparts(self):
        return {self.names["left"]: self.left, self.names["right"]: self.right}

    def materialize(self, make):
        # (runs before the two mixers' own `materialize`: they then find their share of the wide matrix)
        wl, wr = self.left.output_width(), self.right.output_width()
        self.w_o = make("o_proj.weight", ParamDecl((self.hidden_size, wl + wr)))
        self.left.shared_o = self.w_o[:, :wl]
        self.right.shared_o = self.w_o[:, wl:]

    def cache_need(self):
        return self.left.cache_need() or self.right.cache_need()

    def aux_cache_need(self):
        return self.left.aux_cache_need() or self.right.aux_cache_need()

    def state_need(self):
        return self.left.state_need() or self.right.state_need()

    def graph_key(self, ctx):
        return (self.left.graph_key(ctx), self.right.graph_key(ctx))

    def graph_key_group(self):
        return (type(self), self.left.graph_key_group(), self.right.graph_key_group())

    def activation_elems(self):
        return (self.left.activation_elems() + self.right.activation_elems() + self.left.output_width()
                + self.right.output_width() + self.hidden_size)

    def output_projection(self):
        return self.w_o, None

    def forward(self, x, ctx, cache):
        T = x.shape[0]
        wl, wr = self.left.output_width(), self.right.output_width()
        both = ctx.workspace.tokens("parallel.rows", T, wl + wr, x.dtype)
        self.left.forward(x, ctx, cache, project_output=False, out=both[:, :wl], out_scale=self.left_scale)
        self.right.forward(x, ctx, cache, project_output=False, out=both[:, wl:], out_scale=self.right_scale)
        out = ctx.workspace.tokens("mixer.out", T, self.hidden_size, x.dtype)
        linear(both, self.w_o, out)
        return out


@register_mixer("parallel_normed_mixers")
class ParallelNormedMixers(Mixer):
    def __init__(self, hidden_size: int, left, right, eps: float, mult: float = 0.5, names: dict | None = None):
        """`left`, `right`: `MixerSpec`s of mixers that can take their input product from a caller (`SharesInput`) and
        put their output where it says (`forward(..., projected=, out=)`).  `names`: the prefixes of the two mixers'
        tensors behind this mixer's own prefix, and the names of the two norms' weights."""
        super().__init__()
        self.hidden_size, self.eps, self.mult = hidden_size, float(eps), float(mult)
        self.left, self.right = build_mixer(left), build_mixer(right)
        for m in (self.left, self.right):
            if not isinstance(m, SharesInput):
                raise ValueError(f"{type(m).__name__} cannot take its input product from a caller")
        if self.left.cache_need() is not None and self.right.cache_need() is not None:
            raise ValueError("at most one of two mixers side by side keeps pages")
        sl, sr = self.left.state_need(), self.right.state_need()
        self.left_state = 0  # floats of the left mixer's part of the state row, where both keep one
        if sl is not None and sr is not None:
            if len(sl.shape) != 1 or len(sr.shape) != 1 or sl.dtype != sr.dtype:
                raise ValueError("two mixers side by side keep flat state rows of one dtype")
            self.left_state = -(-sl.shape[0] // 4) * 4
        n = dict(left="left.", right="right.", left_norm="left_norm.weight", right_norm="right_norm.weight")
        n.update(names or {})
        self.names = n
        # each side's columns of the input product start on a 16-byte border in every dtype
        self.left_cols = -(-self.left.input_width() // 8) * 8
        self.in_cols = self.left_cols + -(-self.right.input_width() // 8) * 8

    def subparts(self):
        return {self.names["left"]: self.left, self.names["right"]: self.right}

    def param_decls(self):
        H, n = self.hidden_size, self.names
        return {n["left_norm"]: ParamDecl((H,), "norm"), n["right_norm"]: ParamDecl((H,), "norm")}

    def materialize(self, make):
        # (runs before the two mixers' own `materialize`: they then find their shares of the wide matrix)
        super().materialize(make)
        wl, wr, lc = self.left.input_width(), self.right.input_width(), self.left_cols
        self.w_in = make("in_proj.weight", ParamDecl((self.in_cols, self.hidden_size)))
        self.w_in[wl:lc].zero_()
        self.w_in[lc + wr:].zero_()  # (so are the parts of the bias that a mixer leaves out)
        self.b_in = None
        if self.left.input_bias() or self.right.input_bias():
            self.b_in = make("in_proj.bias", ParamDecl((self.in_cols,), "bias"))
            self.b_in.zero_()
        for m, a, n in ((self.left, 0, wl), (self.right, lc, wr)):
            m.shared_in = (self.w_in[a:a + n], self.b_in[a:a + n] if m.input_bias() else None)

    def cache_need(self):
        return self.left.cache_need() or self.right.cache_need()

    def aux_cache_need(self):
        return self.left.aux_cache_need() or self.right.aux_cache_need()

    def state_need(self):
        sl, sr = self.left.state_need(), self.right.state_need()
        if self.left_state:
            return StateNeed((self.left_state + -(-sr.shape[0] // 4) * 4,), sl.dtype)
        return sl or sr

    def graph_key(self, ctx):
        return (self.left.graph_key(ctx), self.right.graph_key(ctx))

    def graph_key_group(self):
        return (type(self), self.left.graph_key_group(), self.right.graph_key_group())

    def operand_dtype(self):
        return self.w_in.dtype

    def activation_elems(self):
        return self.in_cols + self.left.activation_elems() + self.right.activation_elems() + 3 * self.hidden_size

    def _sides(self, x, ctx, cache):
        T, ws = x.shape[0], ctx.workspace
        both = ws.tokens("parallel.in", T, self.in_cols, x.dtype)
        linear(x, self.w_in, both, self.b_in)
        a = ws.tokens("parallel.left", T, self.hidden_size, x.dtype)
        b = ws.tokens("parallel.right", T, self.hidden_size, x.dtype)
        lc = self.left_cols
        left_cache = right_cache = cache
        if self.left_state and cache.state is not None:
            left_cache = replace(cache, state=cache.state[:, :self.left_state])
            right_cache = replace(cache, state=cache.state[:, self.left_state:])
        self.left.forward(x, ctx, left_cache, projected=both[:, :self.left.input_width()], out=a)
        self.right.forward(x, ctx, right_cache, projected=both[:, lc:lc + self.right.input_width()], out=b)
        return a, b

    def forward(self, x, ctx, cache):
        a, b = self._sides(x, ctx, cache)
        out = ctx.workspace.tokens("mixer.out", x.shape[0], self.hidden_size, x.dtype)
        n = self.names
        kernels().pair_norm_add_norm(a, b, self.tensors[n["left_norm"]], self.tensors[n["right_norm"]], self.eps, self.mult,
                                     rows_out=out)
        return out

    def forward_add(self, x, ctx, cache, stream, scale=None, next_norm=None):
        if scale is not None or stream.dtype != torch.float32:
            return False
        a, b = self._sides(x, ctx, cache)
        n = self.names
        kernels().pair_norm_add_norm(a, b, self.tensors[n["left_norm"]], self.tensors[n["right_norm"]], self.eps, self.mult,
                                     stream=stream, next_norm=next_norm)
        return True

    def forward_norm_add(self, x, ctx, cache, stream, norm, mult, copy=None):
        if stream.dtype != torch.float32:
            return False
        a, b = self._sides(x, ctx, cache)
        n = self.names
        kernels().pair_norm_add_norm(a, b, self.tensors[n["left_norm"]], self.tensors[n["right_norm"]], self.eps, self.mult,
                                     stream=stream, next_norm=(None, 0.0, 3, copy) if copy is not None else None,
                                     outer_norm=(*norm, mult))
        return True
