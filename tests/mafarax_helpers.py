"""Small Mafarax configurations for the tests, and model folders and runners made from them."""

from __future__ import annotations

import copy

import torch

import plain_mafarax as pm
from conftest import device
from ludalix_helpers import replay, write_model  # noqa: F401  (step plans replayed through the step function)


def left(heads, kv_heads, dim, vdim, scale, size, rot_dims=None, base=10000.0, factor=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if size is not None:
        m["mask"] = dict(size=size)
    if rot_dims:
        m["rot"] = dict(dims=rot_dims, base=base)
        if factor is not None:
            m["rot"]["scaling"] = dict(factor=factor)
    return m


def right(heads, vdim, state, groups, conv, norm_groups):
    return dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups)


def moe(experts, top, ff, groups=None, scale=1.0, shared=None):
    """`groups`: (count, keep) or None; `shared`: ff or None."""
    r = dict(experts=experts, top=top, scale=scale)
    if groups:
        r["groups"] = dict(count=groups[0], keep=groups[1])
    return dict(kind="moe", expert=dict(ff=ff), router=r, shared=dict(ff=shared) if shared else None)


def config(width, vocab, layers, logit_scale=1.0, eps=2e-6):
    """`layers`: (left, right, mlp) triples."""
    return dict(architecture="Mafarax", vocab=vocab, width=width, logit_scale=logit_scale, norm=dict(eps=eps),
                layers=[dict(type="parallel", mixer=dict(left=a, right=s), mlp=f) for a, s, f in layers])


# A: values wider than keys, a part of each head rotated, stretches of 9; two groups of B and C; three expert groups of
# which two are kept, a shared expert of another size; a layer without feed-forward; one kv head for six heads and a shared
# expert of the experts' own size (it rides in their grouped products)
CFG_A = config(72, 211, [
    (left(4, 2, 24, 40, 0.2, 9, rot_dims=8, base=900.0, factor=3.0), right(4, 12, 20, 2, 4, 2),
     moe(6, 3, 48, groups=(3, 2), scale=1.7, shared=40)),
    (left(2, 2, 16, 16, 0.3, 20, rot_dims=16, base=300.0, factor=0.5), right(2, 24, 16, 1, 3, 1), None),
    (left(6, 1, 16, 8, 0.25, 13, rot_dims=4, base=50.0, factor=2.0), right(6, 8, 12, 3, 2, 4),
     moe(8, 2, 32, groups=(4, 1), scale=0.6, shared=32)),
], logit_scale=0.7)
# B: stretches of 5 under pages of 4; every expert chosen in one layer, groups of a single expert in another; a
# convolution whose memory (6 rows) is longer than most steps
CFG_B = config(64, 97, [
    (left(6, 3, 16, 8, 0.3, 5, rot_dims=4, base=20.0, factor=1.5), right(3, 16, 8, 1, 7, 3), moe(3, 3, 24, shared=16)),
    (left(2, 1, 8, 8, 0.4, 6, rot_dims=8, base=100.0, factor=4.0), right(4, 8, 32, 4, 5, 2),
     moe(4, 2, 40, groups=(4, 3), scale=2.0, shared=40)),
], logit_scale=2.5, eps=1e-5)
# C: sizes that are no multiple of 8 or of 4; stretches of one page and of 3; two experts per group
CFG_C = config(100, 130, [
    (left(4, 4, 36, 20, 0.15, 16, rot_dims=10, factor=2.0), right(3, 5, 7, 1, 4, 5), moe(6, 2, 36, groups=(3, 1), scale=1.1, shared=52)),
    (left(2, 2, 68, 20, 0.06, 3, rot_dims=34, factor=8.0), right(5, 9, 33, 5, 2, 3), moe(3, 2, 44, shared=20)),
    (left(4, 1, 12, 12, 0.3, 7, rot_dims=12, base=7.0, factor=1.2), right(1, 21, 70, 1, 3, 7), None),
], logit_scale=0.3)
# D: values the other three make equal or leave out: one head, stretches of one position, a convolution of one tap (no
# memory), a state of one row, one expert, no shared expert, no mask, no rotation, no scaling of the frequencies, one group
CFG_D = config(48, 61, [
    (left(1, 1, 32, 32, 0.2, 1, rot_dims=2), right(1, 16, 1, 1, 1, 1), moe(1, 1, 32)),
    (left(3, 3, 16, 24, 0.25, None), right(2, 1, 24, 2, 1, 2), moe(4, 1, 24, groups=(1, 1), scale=3.0)),
    (left(2, 1, 15, 9, 0.25, 6, rot_dims=6, base=11.0), right(3, 4, 5, 3, 6, 1), moe(4, 4, 16, groups=(2, 2), shared=8)),
])
# E: sizes the tensor-core kernels of the 16-bit path take: heads of 64 and 128 with stretches longer than a key tile,
# heads of 64 with values of 112, heads of 32 with values of 48; states of 64 and 128 rows
CFG_E = config(96, 150, [
    (left(4, 2, 64, 64, 0.125, 70, rot_dims=32, factor=2.0), right(4, 64, 64, 1, 4, 1), moe(4, 2, 64, groups=(2, 1), shared=64)),
    (left(4, 1, 128, 128, 0.09, 40, rot_dims=64, base=500.0, factor=3.0), right(2, 32, 128, 2, 4, 2), None),
    (left(6, 1, 64, 112, 0.11, 90, rot_dims=48, factor=5.0), right(6, 16, 32, 3, 4, 1), moe(8, 4, 32, groups=(2, 2), scale=1.4, shared=32)),
    (left(2, 2, 32, 48, 0.2, 33, rot_dims=8, factor=1.5), right(2, 128, 16, 1, 4, 2), None),
], logit_scale=0.45)

CONFIGS = {"A": (CFG_A, 8), "B": (CFG_B, 4), "C": (CFG_C, 16), "D": (CFG_D, 8), "E": (CFG_E, 16)}  # config, page size


def cast(w, dtype):
    return w if dtype == "float32" else {n: t.to(getattr(torch, dtype)) for n, t in w.items()}


def weights_for(tag: str, dtype: str, seed: int = 0):
    cfg, page = CONFIGS[tag]
    w = pm.random_weights(cfg, seed=seed + sum(map(ord, tag)))
    return copy.deepcopy(cfg), cast(w, dtype), page


def every_expert_chosen(cfg):
    """The configuration with every expert chosen.  The weights are the same; what falls away is the one discontinuity of
    the design: with a real choice, 16-bit rounding sends a token whose last chosen and first rejected experts (or groups)
    are nearly tied to another expert, and through keys, values and state the difference reaches every later token.
    Whole models in 16-bit are compared in this form; the choice itself is compared in 32-bit (whole models) and in
    16-bit on the feed-forward alone, close calls left out."""
    c = copy.deepcopy(cfg)
    for L in c["layers"]:
        if L["mlp"] is not None:
            r = L["mlp"]["router"]
            r["top"] = r["experts"]
            r.pop("groups", None)
    return c


def model_for(tag: str, dtype: str):
    """(config, weights, page size) of a whole-model comparison: as configured in 32-bit, with every expert chosen in
    16-bit."""
    cfg, w, page = weights_for(tag, dtype)
    return (cfg if dtype == "float32" else every_expert_chosen(cfg)), w, page


def make_runner(tmp_path, cfg, w, page, dtype, num_pages=64, max_requests=4, name="m", **kw):
    from ullm_b200.engine import ModelRunner

    d = write_model(str(tmp_path / f"{name}_{dtype}"), cfg, w)
    return ModelRunner(d, dtype=dtype, device=device(), page_size=page, num_pages=num_pages, max_requests=max_requests,
                       max_context=num_pages * page, max_step_tokens=64, poison_cache=True, **kw)


def oracle(ids, w, cfg) -> torch.Tensor:
    """Logits at every position, 64-bit arithmetic on the weights as given (rounded ones stay rounded)."""
    return pm.forward(cfg, {n: t.double() for n, t in w.items()}, ids).float()
