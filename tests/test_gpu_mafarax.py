"""The Mafarax decoder in the engine against the plain implementation (tests/plain_mafarax.py): each mechanism alone,
whole prompts against token-by-token decoding and portions down to two tokens, unequal batches with pages and request
slots that are used again, the edges of stretches (with weights made so that one key decides), a far key among hundreds,
a state that remembers a token from hundreds of positions back, the first tokens, long decoding, and greedy generation
through the entry point and the scheduler."""

import copy

import pytest
import torch

import plain_mafarax as pm
from conftest import device
from helpers import TOL, TOL_RMS, assert_close, errors, random_ids
from ludalix_helpers import assert_rows_close
from mafarax_helpers import (CONFIGS, cast, config, every_expert_chosen, left, make_runner, model_for, moe, oracle, replay,
                             right, weights_for, write_model)

pytestmark = pytest.mark.gpu


def close(got, ref, dtype, what):
    """A part alone: 32-bit to 3e-5 of the largest value; bfloat16 within the limits the whole models get."""
    if dtype != "float32":
        return assert_close(got, ref, dtype, what)
    mx, _ = errors(got, ref)
    assert torch.isfinite(got.float()).all(), f"{what}: non-finite"
    assert mx <= 3e-5, f"{what}: max err {mx:.2e} of scale"


def rand(shape, seed, dtype, scale=1.0):
    t = torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale
    return t.to(getattr(torch, dtype)).to(device())


def double(w):
    return {n: t.double() for n, t in w.items()}


def mixer_in_steps(r, part, layer, x, cuts):
    """`part` (the mixer of `layer` or one of its two sides) on the rows x, cut into steps at `cuts`."""
    from ullm_b200.engine import StepEntry

    got = []
    r.add_request("a")
    for a, b in zip((0,) + tuple(cuts), tuple(cuts) + (x.shape[0],)):
        e = [StepEntry("a", [0] * (b - a), [])]
        ctx = r.prepare(e)
        caches = r.cache.layer_caches(ctx.groups)
        got.append(part.forward(x[a:b].clone(), ctx, caches[layer]).float().cpu().clone())
        r.commit(e)
    r.check_device_status()
    r.end_request("a")
    return torch.cat(got)


# ---------------------------------------------------------------------------------------------------------
# each mechanism alone
# ---------------------------------------------------------------------------------------------------------
LAYERS = [(tag, i) for tag, (cfg, _) in CONFIGS.items() for i in range(len(cfg["layers"]))]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag,layer", LAYERS)
def test_both_sides_of_every_mixer_and_their_sum(tmp_path, dtype, tag, layer):
    """Random rows in steps of 29, 2, 1, 15, 60 and 3 tokens (stretches of 1 to 90 end inside a portion and between
    portions) against each side and the whole mixer run at once.  The state is zeroed in between: the slot is used
    three times."""
    cfg, w, page = weights_for(tag, dtype)
    r = make_runner(tmp_path, cfg, w, page, dtype)
    x = rand((110, cfg["width"]), 5 + layer, dtype)
    wd, m, eps, pre = double(w), cfg["layers"][layer]["mixer"], cfg["norm"]["eps"], f"l{layer}.mix."
    xd = x.double().cpu()
    cuts = (29, 31, 32, 47, 107)
    mixer = r.model.blocks[layer].mixer
    a = pm.left_mixer(xd, m["left"], wd, pre + "left.")
    b = pm.right_mixer(xd, m["right"], wd, pre + "right.", eps)
    close(mixer_in_steps(r, mixer.left, layer, x, cuts), a.float(), dtype, f"{tag} layer {layer} left")
    # (the right side is divided by its own root mean square: in 16-bit the rows where it nearly vanishes are noisy)
    rows_close = close if dtype == "float32" else assert_rows_close
    rows_close(mixer_in_steps(r, mixer.right, layer, x, cuts), b.float(), dtype, f"{tag} layer {layer} right")
    ref = pm.parallel_mixer(xd, m, wd, pre, eps)
    rows_close(mixer_in_steps(r, mixer, layer, x, cuts), ref.float(), dtype, f"{tag} layer {layer} both")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_mixer_adds_itself_to_the_stream_with_the_next_norms_rows(tmp_path, dtype):
    from ullm_b200.engine import StepEntry

    for tag in ("A", "C", "E"):
        cfg, w, page = weights_for(tag, dtype)
        r = make_runner(tmp_path, cfg, w, page, dtype, name=tag)
        W = cfg["width"]
        x = rand((13, W), 5, dtype)
        wd = double(w)
        stream0 = torch.randn(13, W, generator=torch.Generator().manual_seed(2))
        ref = stream0.double() + pm.parallel_mixer(x.double().cpu(), cfg["layers"][0]["mixer"], wd, "l0.mix.", cfg["norm"]["eps"])
        r.add_request("a")
        ctx = r.prepare([StepEntry("a", [0] * 13, [])])
        stream = stream0.clone().to(device())
        rows = x.clone()  # (the next norm's rows take the input's place)
        block = r.model.blocks[0]
        assert block.mixer.forward_add(rows, ctx, r.cache.layer_caches(ctx.groups)[0], stream, None,
                                       (*block.feed_forward_norm.row_params(), rows))
        close(stream, ref.float(), dtype, f"{tag}: stream")
        close(rows, pm.dynamic_tanh(ref, wd, "l0.norm2").float(), dtype, f"{tag}: next norm")
        r.check_device_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cols", [40, 37, 1024])
def test_tanh_norm_and_pair_norm_kernels(dtype, cols):
    """The tanh norm as the next norm of an addition and over gathered rows; two normed operands added with each kind of
    next norm (RMS, centred, tanh)."""
    from ullm_b200.csrc import kernels

    K, T = kernels(), 11
    td = getattr(torch, dtype)
    g = torch.Generator().manual_seed(cols)
    stream0 = torch.randn(T, cols, generator=g) * 2
    a, b = (torch.randn(T, cols, generator=g).to(td) for _ in range(2))
    wa, wb, w2, b2 = (1 + 0.3 * torch.randn(cols, generator=g) for _ in range(4))
    alpha = torch.tensor(0.6)
    eps = 1e-3
    dev = lambda *ts: [t.to(device()) for t in ts]
    tanh = lambda s: torch.tanh(alpha.double() * s) * w2.double() + b2.double()
    rms = lambda v: v.double() / torch.sqrt((v.double() ** 2).mean(-1, keepdim=True) + eps)
    cen = lambda v: (v - v.mean(-1, keepdim=True)) / torch.sqrt(((v - v.mean(-1, keepdim=True)) ** 2).mean(-1, keepdim=True) + eps)
    sa, da, db, dwa, dwb, dw2, db2, dal = dev(stream0, a, b, wa, wb, w2, b2, alpha)
    out = torch.empty(T, cols, dtype=td, device=device())
    # an operand that is only added, then the tanh norm
    s = sa.clone()
    K.norm_add_norm(s, da, plain=True, next_norm=(dw2, 0.0, 2, dal, db2, out))
    ref = stream0.double() + a.double()
    close(s, ref.float(), "float32", "plain sum")
    close(out, tanh(ref).float(), dtype, "tanh behind a plain sum")
    # gathered rows
    rows = torch.tensor([3, 0, 10, 3], dtype=torch.int32, device=device())
    few = torch.empty(4, cols, dtype=td, device=device())
    K.norm_rows(sa, rows, dw2, 0.0, few, alpha=dal, bias=db2)
    close(few, tanh(stream0.double())[rows.cpu().long()].float(), dtype, "gathered rows")
    # two normed operands
    both = 0.5 * (rms(a) * wa.double() + rms(b) * wb.double())
    for kind, fn, tail in ((0, lambda v: rms(v) * w2.double(), ()), (1, lambda v: cen(v) * w2.double(), ()),
                           (2, tanh, (dal, db2))):
        s = sa.clone()
        K.pair_norm_add_norm(da, db, dwa, dwb, eps, 0.5, stream=s, next_norm=(dw2, eps, kind, *tail, out))
        close(s, (stream0.double() + both).float(), "float32", f"pair sum, kind {kind}")
        close(out, fn(stream0.double() + both).float(), dtype, f"next norm of kind {kind}")
    K.pair_norm_add_norm(da, db, dwa, dwb, eps, 0.5, rows_out=out)
    close(out, both.float(), dtype, "rows without a stream")
    K.raise_on_status()


def test_routing_by_groups_against_the_plain_choice():
    """The routing kernel alone on logits without ties: groups of one, two and many experts, one and several kept, with
    and without further experts that every token takes."""
    from ullm_b200.csrc import kernels

    K = kernels()
    g = torch.Generator().manual_seed(1)
    for E, top, count, keep, always in ((12, 3, 2, 1, 0), (8, 3, 4, 2, 1), (6, 2, 6, 3, 0), (64, 6, 8, 3, 1), (96, 8, 2, 2, 0),
                                        (300, 5, 100, 7, 2), (5, 5, 1, 1, 0), (128, 4, 32, 31, 1)):
        T = 37
        z = torch.randn(T, E + 3, generator=g)  # (further columns behind the experts')
        choice = torch.full((T, top + always), -7, dtype=torch.int32, device=device())
        weight = torch.zeros(T, top + always, device=device())
        K.moe_route(z.to(device()), choice, weight, top, experts=E, groups=count, keep=keep, scale=1.3, always=always)
        w = {"router": torch.eye(E, dtype=torch.float64)}
        ref, rw = pm.route(z[:, :E].double(), w, "", dict(experts=E, top=top, scale=1.3, groups=dict(count=count, keep=keep)))
        assert (choice[:, :top].cpu().long() == ref).all(), (E, top, count, keep)
        assert torch.allclose(weight[:, :top].cpu().double(), rw, rtol=1e-5)
        for j in range(always):
            assert (choice[:, top + j] == E + j).all() and (weight[:, top + j] == 1).all()


@pytest.mark.parametrize("heads,pdim,n,groups", [(2, 16, 32, 1), (4, 32, 64, 2), (3, 64, 128, 1), (2, 48, 256, 2), (40, 64, 128, 1)])
def test_the_chunked_recurrence_against_the_plain_one(heads, pdim, n, groups):
    """Portions of unequal length in one batch (one of them short enough to be left to the token-by-token kernel, one that
    ends on a chunk's edge, one inside), from states that are not zero, with decays from nearly one to nearly nothing: the
    chunked form, the token-by-token kernel and the plain recurrence in 64-bit give the same outputs and states."""
    from ullm_b200.csrc import kernels

    K = kernels()
    lens, least = (130, 5, 64, 77, 192, 17), 16
    T, B = sum(lens), len(lens)
    g = torch.Generator().manual_seed(heads + n)
    inner, ch = heads * pdim, heads * pdim + 2 * groups * n
    xbc = (torch.randn(T, ch, generator=g) * 0.7).to(torch.bfloat16)
    dt = torch.rand(T, heads, generator=g) * 0.5
    dt[::13] *= 10.0
    a = -dt * torch.exp(torch.linspace(-5.0, 2.0, heads))
    D = torch.randn(heads, generator=g)
    slots = [4, 0, 5, 1, 3, 2]
    width = heads * pdim * n + 8
    state0 = torch.randn(B, width, generator=g) * 0.3
    cu = [0]
    for k in lens:
        cu.append(cu[-1] + k)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=device())
    cu_q, req_slots, token_req = i32(cu), i32(slots), i32([i for i, k in enumerate(lens) for _ in range(k)])
    dev = [t.to(device()) for t in (xbc, dt, a, D)]
    ref = torch.zeros(T, inner, dtype=torch.float64)
    ref_state = state0.double().clone()
    for i in range(B):
        S = state0[slots[i], :heads * pdim * n].double().reshape(heads, pdim, n).transpose(1, 2)  # [heads, N, P]
        for t in range(cu[i], cu[i + 1]):
            row = xbc[t].double()
            x = row[:inner].reshape(heads, pdim)
            Bm, Cm = (row[o:o + groups * n].reshape(groups, n).repeat_interleave(heads // groups, 0) for o in (inner, inner + groups * n))
            S = torch.exp(a[t].double())[:, None, None] * S + dt[t].double()[:, None, None] * Bm[:, :, None] * x[:, None, :]
            ref[t] = (torch.einsum("hnp,hn->hp", S, Cm) + D.double()[:, None] * x).reshape(-1)
        ref_state[slots[i], :heads * pdim * n] = S.transpose(1, 2).reshape(-1)
    assert K.ssd_chunk_applies(torch.bfloat16, heads, n, pdim, groups)
    for name in ("chunked", "token by token"):
        state = state0.to(device())
        y = torch.full((T, inner), float("nan"), device=device())
        if name == "chunked":
            scores = torch.full((K.ssd_chunk_floats(T, groups),), float("nan"), device=device())
            K.ssd_chunk(dev[0], inner, inner + groups * n, dev[1], dev[2], dev[3], scores, state, cu_q, req_slots, token_req,
                        y, B, heads, n, pdim, groups, least)
            assert torch.isnan(y[130:135]).all() and not torch.isnan(y[:130]).any() and not torch.isnan(y[135:]).any()
        K.ssd_recurrence(dev[0], inner, inner + groups * n, dev[1], dev[2], dev[3], state, cu_q, req_slots, token_req, y, B,
                         heads, n, pdim, groups, least if name == "chunked" else 1 << 30)
        K.raise_on_status()
        close(y, ref.float(), "float32", f"{name}: outputs")
        close(state, ref_state.float(), "float32", f"{name}: states")


def _ctx_for(r, tokens=128):
    from ullm_b200.engine.batch import Workspace

    class Ctx:
        workspace = Workspace(r.device, max_tokens=tokens, max_requests=4)

    return Ctx()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["A", "B", "C", "D", "E"])
def test_every_feed_forward_alone_and_added_to_the_stream(tmp_path, dtype, tag):
    """Router, groups, ungated experts, the shared expert (riding in the grouped products of few rows, and as products of
    its own beyond them), the sum added to a 32-bit stream with the tanh norm's rows.  Rows whose choice is a close call in
    the plain model do not count in 16-bit."""
    cfg, w, page = weights_for(tag, dtype)
    r = make_runner(tmp_path, cfg, w, page, dtype)
    wd = double(w)
    for T in (21, 90):
        x = rand((T, cfg["width"]), 8 + T, dtype, 1.5)
        stream0 = torch.randn(T, cfg["width"], generator=torch.Generator().manual_seed(4))
        for l, L in enumerate(cfg["layers"]):
            if L["mlp"] is None:
                continue
            pre, f = f"l{l}.mlp.", L["mlp"]
            ff = r.model.blocks[l].feed_forward
            ref = pm.routed_ff(x.double().cpu(), f, wd, pre)
            clear = torch.ones(T, dtype=torch.bool)
            if dtype != "float32":
                rt = f["router"]
                chosen, _ = pm.route(x.double().cpu(), wd, pre, rt)
                g = torch.Generator().manual_seed(3)
                z = x.double().cpu() @ wd[pre + "router"].T
                for _ in range(8):  # a choice that a small disturbance of the logits changes is a close call
                    noisy, _ = pm.route(z + 0.01 * torch.randn(z.shape, generator=g, dtype=torch.float64),
                                        {"router": torch.eye(rt["experts"], dtype=torch.float64)}, "", rt)
                    clear &= (noisy.sort(-1).values == chosen.sort(-1).values).all(-1)
                assert clear.sum() >= T // 2
            got = ff.forward(x.clone(), _ctx_for(r)).float().cpu()
            close(got[clear], ref[clear].float(), dtype, f"{tag} layer {l} feed-forward, {T} rows")
            stream, rows = stream0.clone().to(device()), x.clone()
            assert ff.forward_add(rows, _ctx_for(r), stream, None, (*r.model.final_norm.row_params(), rows))
            s = stream0.double() + ref
            close(stream.cpu()[clear], s[clear].float(), dtype, f"{tag} layer {l} stream, {T} rows")
            close(rows.cpu()[clear], pm.dynamic_tanh(s, wd, "final.norm")[clear].float(), dtype, f"{tag} layer {l} next norm")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_biases_norm_weights_skip_and_scales_each_show(tmp_path, dtype):
    """A model whose biases, slopes, skip weights, side norms and scales are far from what leaves them unseen: whole prompt
    and portions against the plain model, and the plain model itself changes when one is left out."""
    cfg = config(56, 80, [(left(4, 2, 16, 24, 0.25, 7, rot_dims=6, base=40.0, factor=2.5), right(4, 8, 12, 2, 4, 2),
                           moe(4, 2, 24, groups=(2, 1), scale=2.2, shared=16))] * 2, logit_scale=0.2)
    w = pm.random_weights(cfg, seed=33)
    for p in ("l0.", "l1."):
        for n in ("q", "k", "v", "o"):
            w[p + f"mix.left.{n}.b"] = w[p + f"mix.left.{n}.b"] * 4
        w[p + "mix.right.D"] = torch.tensor([2.0, -1.0, 0.5, 3.0])
        w[p + "mix.right.conv.b"] = w[p + "mix.right.conv.b"] * 4
        w[p + "mix.left.out"] = torch.linspace(0.2, 2.0, 56)
        w[p + "mix.right.out"] = torch.linspace(2.0, 0.2, 56)
        w[p + "norm1.b"] = w[p + "norm1.b"] * 3
        w[p + "norm2.alpha"] = torch.tensor(1.5)
    w = cast({n: t.to(torch.bfloat16).float() for n, t in w.items()}, dtype)
    cfg = cfg if dtype == "float32" else every_expert_chosen(cfg)
    ids = random_ids(80, 40, 2)
    ref = oracle(ids, w, cfg)
    for name, val in [(f"l0.mix.left.{n}.b", 0.0) for n in ("qkvo" if dtype == "float32" else "vo")] + [("l0.mix.right.D", 0.0), ("l0.mix.right.conv.b", 0.0),
                      ("l1.mix.left.out", 1.0), ("l0.mix.right.out", 1.0), ("l1.norm1.b", 0.0), ("l1.norm2.alpha", 1.0)]:
        other = dict(w)
        other[name] = torch.full_like(w[name], val)
        assert (oracle(ids, other, cfg) - ref).abs().max() > 3 * TOL[dtype] * ref.abs().max(), name
    r = make_runner(tmp_path, cfg, w, 8, dtype)
    got = replay(r, {"a": ids}, [[("a", 17)], [("a", 2)], [("a", 21)]])["a"]
    assert_rows_close(got, ref, dtype, "biases, norms, skips and scales")


# ---------------------------------------------------------------------------------------------------------
# whole prompts, token-by-token decoding, portions
# ---------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["A", "B", "C", "D", "E"])
def test_whole_decode_and_portions_agree_with_the_plain_model(tmp_path, dtype, tag):
    cfg, w, page = model_for(tag, dtype)
    r = make_runner(tmp_path, cfg, w, page, dtype, num_pages=64)
    n = 75 if tag != "E" else 190  # (E: stretches of 70 and 90 must end in prompts and among decoded tokens)
    ids = random_ids(cfg["vocab"], n, 11)
    ref = oracle(ids, w, cfg)
    plans = {
        "whole": [[("a", n)]],
        "decode": [[("b", 3)]] + [[("b", 1)] for _ in range(n - 3)],
        "portions": [[("c", k)] for k in (2, 2, 3, 7, 2, 16, 1, 1, 2, 31, 8) + ((70, 2, 43) if n == 190 else ())],
        "one by one": [[("d", 1)] for _ in range(n)],
    }
    assert sum(k for (_, k), in plans["portions"]) == n
    for name, plan in plans.items():
        rid = plan[0][0][0]
        got = replay(r, {rid: ids}, plan)[rid]
        assert_rows_close(got, ref, dtype, f"{tag} {name}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["A", "E"])
def test_unequal_batches_with_pages_and_slots_used_again(tmp_path, dtype, tag):
    """Three request slots and a pool that cannot hold all requests at once: six requests of unequal length come
    and go, portions of some beside single tokens of others; every request equals itself run alone."""
    cfg, w, page = model_for(tag, dtype)
    pages = 24 if tag == "A" else 17
    r = make_runner(tmp_path, cfg, w, page, dtype, num_pages=pages, max_requests=3)
    lens = dict(a=50, b=9, c=61, d=2, e=33, f=17)
    reqs = {k: random_ids(cfg["vocab"], n, 40 + n) for k, n in lens.items()}
    plan = [
        [("a", 20), ("b", 2)],
        [("a", 1), ("b", 5), ("c", 30)],
        [("b", 2), ("a", 9), ("c", 1)],          # b ends: its slot and pages go back
        [("d", 2), ("c", 1), ("a", 1)],          # d takes them, and ends at once
        [("e", 16), ("a", 19)],                  # a ends
        [("c", 29), ("e", 1), ("f", 2)],         # c ends; f starts on a slot and pages that were used
        [("f", 15), ("e", 16)],
    ]
    got = replay(r, reqs, plan)
    for k in reqs:
        assert_rows_close(got[k], oracle(reqs[k], w, cfg), dtype, f"request {k}")
    assert not r.cache.requests
    assert all(r.cache.num_free_pages(g) == n for g, n in enumerate(r.cache.group_pages))


# ---------------------------------------------------------------------------------------------------------
# edges: stretches of positions, page borders; weights made so that one key decides
# ---------------------------------------------------------------------------------------------------------
def one_key_model(size, dtype, dim, vdim, heads=2, kv_heads=1):
    """One layer without feed-forward whose queries are scaled up: the softmax is nearly one-hot, so a key that is wrongly
    seen or wrongly hidden changes the logits by much more than any tolerance."""
    sharp = 4.0 if dtype == "float32" else 2.5
    cfg = config(48, 61, [(left(heads, kv_heads, dim, vdim, 1.0 / dim ** 0.5, size, rot_dims=4, base=1e6), right(2, 8, 8, 1, 2, 1), None)])
    w = pm.random_weights(cfg, seed=size * 31 + dim)
    w["l0.mix.left.q"] = (w["l0.mix.left.q"] * sharp).to(torch.bfloat16).float()
    w["l0.mix.right.out"] = w["l0.mix.right.out"] * 0.25
    return cfg, cast(w, dtype)


def with_stretch(cfg, size):
    c = copy.deepcopy(cfg)
    c["layers"][0]["mixer"]["left"]["mask"] = dict(size=size)
    return c


EDGES = [(8, 32, 32), (4, 64, 64), (70, 64, 64), (5, 128, 128), (17, 24, 40), (9, 32, 48), (66, 128, 128), (33, 48, 16),
         (100, 64, 112), (64, 64, 64)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size,dim,vdim", EDGES)
def test_stretch_edges_in_prompts_and_decoding(tmp_path, dtype, size, dim, vdim):
    page = 8
    cfg, w = one_key_model(size, dtype, dim, vdim)
    n = 70 if size < 30 else 2 * size + 12  # (an edge among the decoded tokens, and one inside the portions)
    # the test has power: a stretch one token longer or shorter is far off (the first of a few token sequences for
    # which both are)
    for seed in range(5, 25):
        ids = random_ids(cfg["vocab"], n, seed)
        ref = oracle(ids, w, cfg)
        offs = [float((oracle(ids, w, with_stretch(cfg, s)) - ref).abs().max() / ref.abs().max()) for s in (size + 1, size - 1)]
        if min(offs) > 5 * TOL[dtype]:
            break
    else:
        raise AssertionError(f"no token sequence makes every edge decisive (last: {offs})")
    r = make_runner(tmp_path, cfg, w, page, dtype, num_pages=20 if size < 100 else 40)
    # portions that end on, one before and one after page borders and edges; then single tokens
    first = (7, 1, 1, 8, 9, 2, 3) if size < 30 else (7, 1, 1, size - 10, 2, 8)
    plan = [[("a", k)] for k in first]
    plan += [[("a", 1)] for _ in range(n - sum(first))]
    got = replay(r, {"a": ids}, plan)["a"]
    whole = replay(r, {"b": ids}, [[("b", n)]])["b"]
    what = f"stretches of {size}, heads of {dim} / {vdim}"
    for name, g in (("cut", got), ("whole", whole)):
        if dtype == "float32":
            assert_close(g, ref, dtype, f"{what}, {name}")
            continue
        # sharp queries multiply the rounding of the 16-bit queries and keys; the largest error stays a quarter of
        # what the nearest wrong edge would cause, the mean error inside the models' limit
        mx, rms = errors(g, ref)
        assert torch.isfinite(g.float()).all(), f"{what}: non-finite logits"
        assert mx <= max(TOL[dtype], min(offs) / 4) and rms <= TOL_RMS[dtype], (
            f"{what}, {name}: max err {mx:.3e} of scale (a wrong edge: {min(offs):.3e}), rms {rms:.3e}")
    assert all(r.cache.num_free_pages(g) == n for g, n in enumerate(r.cache.group_pages))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,vdim", [(24, 20), (64, 112), (128, 128)])
def test_a_far_key_among_hundreds_decides(tmp_path, dtype, dim, vdim):
    """Stretches of 500: at the end of 400 tokens the asking token's query matches the key of ONE marked token near the
    start, and the logits say which token stood there.  The asking token's query is made to point at the marked token's
    key (a rank-one W_q on its normed embedding)."""
    H = 2
    cfg = config(48, 61, [(left(H, 1, dim, vdim, 1.0, 500), right(2, 8, 8, 1, 2, 1), None)])
    w = pm.random_weights(cfg, seed=dim)
    asks, marked, other = 58, 60, 59
    wd = double(w)
    h = lambda tok: pm.dynamic_tanh(wd["embed"][tok], wd, "l0.norm1")
    key = wd["l0.mix.left.k"] @ h(marked) + wd["l0.mix.left.k.b"]
    sharp = 30.0
    wq = sharp * key[:, None] * h(asks)[None, :] / float(h(asks) @ h(asks)) / float(key @ key)
    w["l0.mix.left.q"] = wq.repeat(H, 1).to(torch.bfloat16).float()
    w["l0.mix.left.q.b"] = torch.zeros(H * dim)
    w["l0.mix.right.out"] = w["l0.mix.right.out"] * 0.125
    w = cast(w, dtype)
    n = 400
    ids = [t % 58 for t in random_ids(61, n, 3)]
    ids[13] = marked
    ids[-1] = asks
    ref = oracle(ids, w, cfg)
    changed = list(ids)
    changed[13] = other
    assert (oracle(changed, w, cfg)[-1] - ref[-1]).abs().max() > 5 * TOL[dtype] * ref.abs().max(), "token 13 must matter"
    r = make_runner(tmp_path, cfg, w, 8, dtype, num_pages=56)
    plan = [[("a", 64)] for _ in range(5)] + [[("a", 2)] for _ in range(20)] + [[("a", 1)] for _ in range(40)]
    got = replay(r, {"a": ids}, plan)["a"]
    assert_close(got[-1:], ref[-1:], dtype, "far key, last row")
    assert_rows_close(got, ref, dtype, "far key")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,vdim,state,groups", [(2, 8, 12, 1), (4, 64, 64, 2), (2, 32, 128, 1)])
def test_the_state_remembers_over_portions_and_single_tokens(tmp_path, dtype, heads, vdim, state, groups):
    """Decays of nearly one: a token 250 positions back still shows in the logits, over stretches of 4 positions that the
    attention forgets at once.  A lost, doubled or mixed-up state would be far off."""
    cfg = config(48, 61, [(left(2, 1, 8, 8, 0.3, 4, rot_dims=4), right(heads, vdim, state, groups, 3, 1), None)])
    w = pm.random_weights(cfg, seed=state)
    w["l0.mix.right.A_log"] = torch.full((heads,), -7.0)
    w["l0.mix.left.out"] = w["l0.mix.left.out"] * 0.125
    w["l0.mix.right.D"] = w["l0.mix.right.D"] * 0.125
    # the marked token's step is large (its row of dt), everyone else's small; B and C have a common direction
    wd = double(w)
    inner = heads * vdim
    marked, other = 60, 59
    h = lambda tok: pm.dynamic_tanh(wd["embed"][tok], wd, "l0.norm1")
    rows = inner + inner + 2 * groups * state
    w["l0.mix.right.conv.b"][inner:] = 1.5
    w["l0.mix.right.in"][rows:] = (16.0 * h(marked) / (h(marked) @ h(marked))).to(torch.bfloat16).float()
    w["l0.mix.right.dt_bias"] = torch.full((heads,), -8.0)
    w = cast(w, dtype)
    n = 290
    ids = [t % 58 for t in random_ids(61, n, 3)]
    ids[30] = marked
    ref = oracle(ids, w, cfg)
    changed = list(ids)
    changed[30] = other
    gone = oracle(changed, w, cfg)
    assert (gone[-1] - ref[-1]).abs().max() > 3 * TOL[dtype] * ref.abs().max(), "token 30 must matter at the end"
    r = make_runner(tmp_path, cfg, w, 8, dtype, num_pages=56)
    for name, plan in (("portions", [64, 2, 2, 100, 2, 64, 1, 3, 2]), ("decode", [40]), ("whole", [n])):
        plan = [[(name, k)] for k in plan]
        plan += [[(name, 1)] for _ in range(n - sum(k for (_, k), in plan))]
        got = replay(r, {name: ids}, plan)[name]
        assert_close(got[-1:], ref[-1:], dtype, f"memory, {name}, last row")
        assert_rows_close(got, ref, dtype, f"memory, {name}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_first_tokens_alone_and_in_pairs(tmp_path, dtype):
    """Requests of one, two and three tokens, each alone in a step and side by side: the first positions (angle 0, a
    softmax over one key, a convolution over zeros, an empty state) against the plain model."""
    for tag in ("A", "B", "D"):
        cfg, w, page = model_for(tag, dtype)
        r = make_runner(tmp_path, cfg, w, page, dtype, name=tag)
        reqs = {k: random_ids(cfg["vocab"], n, 7 + n) for k, n in dict(a=1, b=2, c=3, d=2).items()}
        got = replay(r, reqs, [[("a", 1)], [("b", 2), ("c", 1)], [("c", 2), ("d", 1)], [("d", 1)]])
        for k in reqs:
            assert_rows_close(got[k], oracle(reqs[k], w, cfg), dtype, f"{tag} request {k}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(tmp_path, dtype):
    """One prompt token, then 300 tokens one by one: stretches end among decoded tokens, pages come and go, the state is
    carried 300 times."""
    cfg, w, page = model_for("B", dtype)
    r = make_runner(tmp_path, cfg, w, page, dtype, num_pages=160)
    ids = random_ids(cfg["vocab"], 301, 17)
    got = replay(r, {"a": ids}, [[("a", 1)] for _ in range(301)])["a"]
    assert_rows_close(got, oracle(ids, w, cfg), dtype, "long decoding")


# ---------------------------------------------------------------------------------------------------------
# generation through the entry point and the scheduler
# ---------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("eager", [True, False])
@pytest.mark.parametrize("tag", ["A", "C"])
def test_greedy_generation_through_the_entry_point(tmp_path, tag, eager):
    """Five prompts under a token budget of 16 and three request slots (prompts are cut into portions, requests
    wait for a slot, decode steps are replayed from CUDA graphs unless eager), greedy, against the plain model
    run on the growing sequence.  A step's choice is compared only where the plain model's margin is clear."""
    from ullm_b200 import LLM, EngineConfig, SamplingParams

    cfg, w, page = weights_for(tag, "float32")
    d = write_model(str(tmp_path / f"gen{tag}{eager}"), cfg, w)
    ec = EngineConfig(model=d, max_bs=3, context_len=128, page_size=page, num_pages=48, max_num_batched_tokens=16,
                      dtype="float32", enforce_eager=eager)
    llm = LLM(ec)
    prompts = [random_ids(cfg["vocab"], n, 90 + n) for n in (1, 6, 23, 40, 17)]
    outs = llm.generate_batch(prompts, SamplingParams(temperature=0.0, max_new_tokens=14, ignore_eos=True))
    wd = double(w)
    for p, o in zip(prompts, outs):
        assert len(o.token_ids) == 14
        seq = list(p)
        for tok in o.token_ids:
            lg = pm.forward(cfg, wd, seq)[-1]
            top2 = torch.topk(lg, 2).values
            if top2[0] - top2[1] > 1e-3 * lg.abs().max():
                assert tok == int(torch.argmax(lg)), f"prompt of {len(p)}: token {len(seq) - len(p)} differs"
            seq.append(tok)
    llm.engine.runner.cache.check_invariants()
