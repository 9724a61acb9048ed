"""Small Ninelix configurations for the tests, and model folders and runners made from them."""

from __future__ import annotations

import copy

import torch

import plain_ninelix as pn
from conftest import device
from ludalix_helpers import replay, write_model  # noqa: F401  (step plans replayed through the step function)


def left(heads, kv_heads, dim, vdim, scale, conv, bias_max, coef=0.4, every=16):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, conv=conv, bias_max=bias_max,
                q_temp=dict(coef=coef, every=every))


def right(heads, vdim, state, groups, conv, norm_groups):
    return dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups)


def parallel(a, s, mlp=None):
    return dict(type="parallel", mixer=dict(left=a, right=s), mlp=mlp)


def wkv(heads, dim, mlp=None):
    return dict(type="wkv", mixer=dict(heads=heads, dim=dim), mlp=mlp)


def lightning(dim, vdim, decay, mlp=None):
    return dict(type="lightning", mixer=dict(heads=len(decay), dim=dim, vdim=vdim, decay=list(decay)), mlp=mlp)


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))


def config(width, vocab, layers, logit_scale=1.0, eps=2e-6, buckets=37, mul_prev=5, mul_cur=3):
    return dict(architecture="Ninelix", vocab=vocab, width=width, logit_scale=logit_scale, norm=dict(eps=eps),
                embedding=dict(bigram=dict(buckets=buckets, mul_prev=mul_prev, mul_cur=mul_cur)), layers=copy.deepcopy(layers))


# A: every kind of layer with every kind of feed-forward, sizes that are multiples of 4 and 8
CFG_A = config(72, 211, [
    parallel(left(4, 2, 24, 40, 0.2, 3, 20, every=7), right(4, 12, 20, 2, 4, 2), moe(6, 3, 48)),
    wkv(3, 24, dense(80)),
    lightning(20, 28, [0.9, 0.5], None),
    wkv(2, 16, moe(5, 2, 40)),
    lightning(16, 16, [1.0, 0.97, 0.2], moe(4, 1, 24)),
    parallel(left(6, 1, 16, 8, 0.3, 2, 60, coef=0.9, every=3), right(2, 24, 16, 1, 3, 1), dense(56)),
], logit_scale=0.7)
# B: a wkv layer first, no feed-forward behind attention, long convolutions whose memories outlast most steps, pages of 4
CFG_B = config(64, 97, [
    wkv(4, 8, None),
    parallel(left(6, 3, 16, 8, 0.3, 6, 9, coef=-0.2, every=5), right(3, 16, 8, 1, 7, 3), None),
    lightning(8, 40, [0.8, 0.99, 0.999, 0.3], dense(48)),
    wkv(1, 40, dense(24)),
], logit_scale=2.5, eps=1e-5, buckets=101, mul_prev=1, mul_cur=10)
# C: sizes that are no multiple of 4 or 8
CFG_C = config(100, 130, [
    lightning(13, 21, [0.7, 0.95, 0.999], dense(35)),
    parallel(left(4, 4, 36, 20, 0.15, 4, 33), right(3, 5, 7, 1, 4, 5), moe(6, 2, 36)),
    wkv(3, 18, moe(3, 2, 52)),
    parallel(left(3, 1, 15, 9, 0.25, 5, 14, coef=1.3, every=1), right(5, 9, 33, 5, 2, 3), None),
    wkv(5, 7, dense(30)),
], logit_scale=0.3, buckets=7, mul_prev=11, mul_cur=4)
# D: values the other ones leave out: one head, convolutions of one tap (no memory), a state of one row, one expert, one
# bucket, no temperature
CFG_D = config(48, 61, [
    parallel(left(1, 1, 32, 32, 0.2, 1, 2, coef=0.0, every=1000), right(1, 16, 1, 1, 1, 1), moe(1, 1, 32)),
    wkv(1, 1, dense(8)),
    lightning(1, 1, [0.5], moe(4, 4, 16)),
    parallel(left(3, 3, 16, 24, 0.25, 1, 5), right(2, 1, 24, 2, 3, 2), dense(16)),
], buckets=1)
# E, F: sizes the tensor-core kernels of the 16-bit path take, distances beyond a key tile
CFG_E = config(96, 150, [
    lightning(64, 48, [0.97, 0.6], dense(64)),
    parallel(left(4, 2, 64, 64, 0.125, 4, 100, every=50), right(4, 64, 64, 1, 4, 1), moe(4, 2, 64)),
    wkv(2, 64, dense(96)),
    parallel(left(6, 1, 64, 112, 0.11, 3, 150, every=40), right(6, 16, 32, 3, 4, 1), None),
], logit_scale=0.45, eps=1e-5)
CFG_F = config(128, 90, [
    wkv(3, 32, None),
    lightning(32, 32, [0.999, 0.9, 0.8], moe(8, 4, 32)),
    parallel(left(2, 1, 128, 128, 0.09, 4, 70, every=30), right(2, 32, 128, 2, 4, 2), None),
    wkv(1, 128, moe(2, 1, 64)),
], logit_scale=1.5, buckets=1009, mul_prev=4001, mul_cur=77)

CONFIGS = {"A": (CFG_A, 8), "B": (CFG_B, 4), "C": (CFG_C, 16), "D": (CFG_D, 8), "E": (CFG_E, 16), "F": (CFG_F, 16)}  # config, page size
# sizes that tensors alone give: ranks of the decays and rows of the distance tables, per layer
TENSOR_SIZES = {
    "A": dict(decay_rank=[0, 8, 0, 24, 0, 0], bias_rows=[10, 0, 0, 0, 0, 32]),
    "B": dict(decay_rank=[40, 0, 0, 3], bias_rows=[0, 6, 0, 0]),
    "C": dict(decay_rank=[0, 0, 5, 0, 70], bias_rows=[0, 9, 0, 4, 0]),
    "D": dict(decay_rank=[0, 1, 0, 0], bias_rows=[2, 0, 0, 3]),
    "E": dict(decay_rank=[0, 0, 32, 0], bias_rows=[0, 24, 0, 32]),
    "F": dict(decay_rank=[16, 0, 0, 200], bias_rows=[0, 0, 12, 0]),
}


def cast(w, dtype):
    return w if dtype == "float32" else {n: t.to(getattr(torch, dtype)) for n, t in w.items()}


def weights_for(tag: str, dtype: str, seed: int = 1):
    """(Seeds whose 16-bit errors are those of rounding alone: a read-out that happens to vanish is divided by its own root
    mean square, and its direction is then a matter of the last bit.)"""
    cfg, page = CONFIGS[tag]
    w = pn.random_weights(cfg, seed=seed + sum(map(ord, tag)), **TENSOR_SIZES[tag])
    return copy.deepcopy(cfg), cast(w, dtype), page


def every_expert_chosen(cfg):
    """The configuration with every expert chosen (the weights are the same).  The choice is the design's one discontinuity:
    in 16-bit a token whose last chosen and first rejected experts are nearly tied may go to another expert, and through
    keys, values and state the difference reaches every later token.  Whole models in 16-bit are compared in this form; the
    choice itself is compared in 32-bit (whole models) and in 16-bit on the feed-forward alone, close calls left out."""
    c = copy.deepcopy(cfg)
    for L in c["layers"]:
        if L["mlp"] is not None and L["mlp"]["kind"] == "moe":
            L["mlp"]["router"]["top"] = L["mlp"]["router"]["experts"]
    return c


def model_for(tag: str, dtype: str):
    """(config, weights, page size) of a whole-model comparison."""
    cfg, w, page = weights_for(tag, dtype)
    return (cfg if dtype == "float32" else every_expert_chosen(cfg)), w, page


def make_runner(tmp_path, cfg, w, page, dtype, num_pages=64, max_requests=4, name="m", **kw):
    from ullm_b200.engine import ModelRunner

    d = write_model(str(tmp_path / f"{name}_{dtype}"), cfg, w)
    return ModelRunner(d, dtype=dtype, device=device(), page_size=page, num_pages=num_pages, max_requests=max_requests,
                       max_context=num_pages * page, max_step_tokens=64, poison_cache=True, **kw)


def oracle(ids, w, cfg) -> torch.Tensor:
    """Logits at every position, 64-bit arithmetic on the weights as given (rounded ones stay rounded)."""
    return pn.forward(cfg, {n: t.double() for n, t in w.items()}, ids).float()


def assert_model_close(got, ids, w, cfg, dtype: str, what: str = "") -> None:
    """A whole model's logits at every position against the plain model.  32-bit: the fixed limits of tests/helpers.py.
    16-bit: a read-out that nearly vanishes is divided by its own root mean square, and every sub-layer's output is normed
    once more, so roundings are amplified at some positions; how far is taken from the plain model with nothing but its
    sub-layers' inputs and outputs rounded, or moved by as much at random (the largest of five runs).  Rows may err by the fixed rms limit or three times that model's own error, there
    or over all rows (one in 25 by twice as much), all rows together by the fixed rms limit or twice its error."""
    from helpers import TOL_RMS, assert_close

    ref = oracle(ids, w, cfg)
    if dtype == "float32":
        return assert_close(got, ref, dtype, what)
    assert got.shape == ref.shape and torch.isfinite(got.float()).all(), f"{what}: shape or non-finite values"
    wd, td = {n: t.double() for n, t in w.items()}, getattr(torch, dtype)
    g = torch.Generator().manual_seed(1)
    unit = torch.finfo(td).eps / 2  # (the largest relative error of a rounding)
    moved = lambda v: v * (1.0 + unit * (2.0 * torch.rand(v.shape, generator=g, dtype=v.dtype) - 1.0))
    own = [pn.forward(cfg, wd, ids, rounded=r).float() - ref for r in [lambda v: v.to(td).double()] + [moved] * 4]
    scale = max(ref.abs().max().item(), 1e-6)
    rms = lambda d: d.pow(2).mean(-1).sqrt() / scale
    err, floor = rms(got.detach().float().cpu() - ref), torch.stack([rms(d) for d in own]).amax(0)
    own_all = float(floor.pow(2).mean().sqrt())
    limit = (3 * floor).clamp(min=max(3 * own_all, TOL_RMS[dtype]))
    total, allowed = err.pow(2).mean().sqrt(), max(TOL_RMS[dtype], 2 * own_all)
    over = int((err > limit).sum())
    assert total <= allowed, f"{what}: rms {total:.3e} (limit {allowed:.3e}) of scale"
    assert over <= max(1, len(err) // 25) and (err <= 2 * limit).all(), (
        f"{what}: {over} of {len(err)} rows over their limit, worst {float((err / limit).max()):.2f} times")
