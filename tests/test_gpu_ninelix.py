"""The Ninelix decoder in the engine against the plain implementation (tests/plain_ninelix.py): each mechanism alone, whole
prompts against token-by-token decoding and portions down to two tokens, unequal batches with pages and request slots that
are used again, the edges of distance buckets (with weights made so that one bucket decides), a far key among hundreds, states
that remember one token from hundreds of positions back, the first tokens, long decoding, and greedy generation through the
entry point and the scheduler."""

import copy
import os
from types import SimpleNamespace

import pytest
import torch

import plain_ninelix as pn
from conftest import device
from helpers import TOL, assert_close, errors, random_ids
from ludalix_helpers import assert_rows_close
from ninelix_helpers import (CONFIGS, assert_model_close, cast, config, dense, every_expert_chosen, left, lightning, make_runner,
                             model_for, moe, oracle, parallel, replay, right, weights_for, wkv, write_model)

pytestmark = [pytest.mark.gpu, pytest.mark.needs_cuda]


def close(got, ref, dtype, what, limit=3e-5):
    """A part alone: 32-bit to 3e-5 of the largest value; bfloat16 within the limits the whole models get."""
    if dtype != "float32":
        return assert_close(got, ref, dtype, what)
    mx, _ = errors(got, ref)
    assert torch.isfinite(got.float()).all(), f"{what}: non-finite"
    assert mx <= limit, f"{what}: max err {mx:.2e} of scale"


def rand(shape, seed, dtype, scale=1.0):
    t = torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale
    return t.to(getattr(torch, dtype)).to(device())


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=device())


def double(w):
    return {n: t.double() for n, t in w.items()}


def in_steps(r, x, cuts, run):
    """`run(rows, ctx, caches)` on the rows x cut into steps at `cuts`, one request; the results one behind the other."""
    from ullm_b200.engine import StepEntry

    got = []
    r.add_request("a")
    for a, b in zip((0,) + tuple(cuts), tuple(cuts) + (x.shape[0],)):
        e = [StepEntry("a", [0] * (b - a), [])]
        ctx = r.prepare(e)
        got.append(run(x[a:b].clone(), ctx, r.cache.layer_caches(ctx.groups)).float().cpu().clone())
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
def test_every_mixer_alone(tmp_path, dtype, tag, layer):
    """Random rows in steps of 29, 2, 1, 15, 60 and 3 tokens against the mixer run at once.  The state is zeroed in between:
    the slot is used again."""
    cfg, w, page = weights_for(tag, dtype)
    r = make_runner(tmp_path, cfg, w, page, dtype)
    x = rand((110, cfg["width"]), 5 + layer, dtype)
    wd, L, eps, pre = double(w), cfg["layers"][layer], cfg["norm"]["eps"], f"l{layer}.mix."
    xd = x.double().cpu()
    m = r.model.blocks[layer].mixer
    what = f"{tag} layer {layer} ({L['type']})"
    # (a read-out that nearly vanishes is divided by its own root mean square: in 16-bit such rows are noisy)
    rows_close = close if dtype == "float32" else assert_rows_close
    if dtype == "bfloat16" and tag == "D" and L["type"] != "parallel":
        return  # (heads of one number: nothing but signs behind the norm)
    for name, cuts in (("steps", (29, 31, 32, 47, 107)), ("whole", ())):
        got = in_steps(r, x, cuts, lambda rows, ctx, caches: m.forward(rows, ctx, caches[layer]))
        rows_close(got, pn.mixer(xd, L, wd, pre, eps).float(), dtype, f"{what}, {name}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_both_sides_of_a_parallel_mixer(tmp_path, dtype):
    for tag, layer in (("A", 0), ("A", 5), ("B", 1), ("C", 1), ("E", 3)):
        cfg, w, page = weights_for(tag, dtype)
        r = make_runner(tmp_path, cfg, w, page, dtype, name=f"{tag}{layer}")
        x = rand((70, cfg["width"]), layer, dtype)
        wd, mx, eps, pre = double(w), cfg["layers"][layer]["mixer"], cfg["norm"]["eps"], f"l{layer}.mix."
        m = r.model.blocks[layer].mixer
        from dataclasses import replace

        n = m.left_state

        def run(part, a, b):
            return lambda rows, ctx, caches: part.forward(rows, ctx, replace(caches[layer], state=caches[layer].state[:, a:b]))

        got = in_steps(r, x, (20, 21, 23, 60), run(m.left, 0, n))
        close(got, pn.left_mixer(x.double().cpu(), mx["left"], wd, pre + "left.", eps).float(), dtype, f"{tag} {layer} left")
        got = in_steps(r, x, (20, 21, 23, 60), run(m.right, n, None))
        rows_close = close if dtype == "float32" else assert_rows_close
        rows_close(got, pn.right_mixer(x.double().cpu(), mx["right"], wd, pre + "right.", eps).float(), dtype, f"{tag} {layer} right")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sub_layers_norm_their_output_and_add_it_to_the_stream(tmp_path, dtype):
    """A block alone: stream and its rounded copy behind mixer and feed-forward, fused into the mixer's and the experts' last
    kernels where they offer it."""
    for tag in ("A", "C", "E", "F"):
        cfg, w, page = weights_for(tag, dtype)
        r = make_runner(tmp_path, cfg, w, page, dtype, name=tag)
        W, wd, eps = cfg["width"], double(w), cfg["norm"]["eps"]
        for layer, L in enumerate(cfg["layers"]):
            if dtype != "float32" and L["mlp"] is not None and L["mlp"]["kind"] == "moe":
                continue  # (the choice reads a rounded stream: compared in 32-bit)
            stream0 = torch.randn(13, W, generator=torch.Generator().manual_seed(layer))
            ref = pn.layer(stream0.double(), layer, cfg, wd)

            def run(rows, ctx, caches):
                ctx.stream_operand, ctx.shared = None, {}
                out = r.model.blocks[layer].forward(rows, None, ctx, caches[layer])
                assert out[0] is None and out[1].data_ptr() == rows.data_ptr()
                copy = ctx.stream_operand
                assert copy.dtype == getattr(torch, dtype) and torch.equal(copy, rows.to(copy.dtype))
                return rows

            rows_close = close if dtype == "float32" else assert_rows_close
            rows_close(in_steps(r, stream0.to(device()), (), run), ref.float(), dtype, f"{tag} layer {layer}")


def _ctx_for(r, tokens=128):
    from ullm_b200.engine.batch import Workspace

    class Ctx:
        workspace = Workspace(r.device, max_tokens=tokens, max_requests=4)

    return Ctx()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["A", "B", "C", "D", "E", "F"])
def test_every_feed_forward_alone(tmp_path, dtype, tag):
    """Exact gelu and routed experts.  Rows whose choice is a close call in the plain model do not count in 16-bit."""
    cfg, w, page = weights_for(tag, dtype)
    r = make_runner(tmp_path, cfg, w, page, dtype)
    wd = double(w)
    for T in (5, 90):
        x = rand((T, cfg["width"]), 8 + T, dtype, 1.5)
        for l, L in enumerate(cfg["layers"]):
            f, pre = L["mlp"], f"l{l}.mlp."
            if f is None:
                assert r.model.blocks[l].feed_forward is None
                continue
            ref = pn.feed_forward(x.double().cpu(), f, wd, pre)
            clear = torch.ones(T, dtype=torch.bool)
            if dtype != "float32" and f["kind"] == "moe" and f["router"]["top"] < f["router"]["experts"]:
                z = (x.double().cpu() @ wd[pre + "router"].T).sort(-1, descending=True).values
                clear = z[:, f["router"]["top"] - 1] - z[:, f["router"]["top"]] > 0.03
            got = r.model.blocks[l].feed_forward.forward(x.clone(), _ctx_for(r)).float().cpu()
            close(got[clear], ref[clear].float(), dtype, f"{tag} layer {l} {f['kind']}, {T} rows")


def test_the_choice_goes_by_logits_where_a_softmax_underflows():
    from ullm_b200.csrc import kernels

    K = kernels()
    z = torch.tensor([[200.0, -1.0, 3.0, 2.0, -300.0, 1.0], [-500.0, -400.0, -450.0, 0.0, -420.0, -410.0]])
    choice = torch.zeros(2, 3, dtype=torch.int32, device=device())
    weight = torch.zeros(2, 3, device=device())
    K.moe_route(z.to(device()), choice, weight, 3, softmax_scores=True, renormalize=True)
    assert choice.tolist() == [[0, 2, 3], [3, 1, 5]]
    assert torch.allclose(weight.cpu(), torch.tensor([[1.0, 0.0, 0.0]] * 2))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("hidden,buckets,mp,mc", [(40, 7, 11, 4), (37, 1, 1, 1), (64, 50021, 1000003, 7919)])
def test_pair_embedding_over_steps(dtype, hidden, buckets, mp, mc):
    """Three requests side by side over several steps, one token and many at a time, the sampled token taken from the device,
    a padding row, and a slot that starts anew."""
    from ullm_b200.csrc import kernels

    K, td = kernels(), getattr(torch, dtype)
    g = torch.Generator().manual_seed(hidden)
    V = 90
    e = torch.randn(V, hidden, generator=g).to(td)
    b = torch.randn(buckets + 1, hidden, generator=g).to(td)
    state = torch.zeros(5, 1, dtype=torch.int32, device=device())
    last = i32([3, 14, 15, 9, 26])
    cfg = dict(embedding=dict(bigram=dict(buckets=buckets, mul_prev=mp, mul_cur=mc)))
    seqs = {s: random_ids(V, 20, s) for s in (4, 0, 2)}
    seqs[2][12] = 15
    at = {s: 0 for s in seqs}
    w = dict(embed=e.double(), bigram=b.double())
    for plan in ([(4, 3), (0, 1)], [(2, 5), (4, 1), (0, 2)], [(0, 1), (4, 1), (2, 1)], [(2, 6)], [(4, 2), (2, "last")]):
        ids, cu, req, slots, want = [], [0], [], [], []
        for r_, (s, n) in enumerate(plan):
            k = 1 if n == "last" else n
            ids += [-1] if n == "last" else seqs[s][at[s]:at[s] + k]
            want.append(pn.embed(seqs[s][:at[s] + k], w, cfg)[at[s]:])
            at[s] += k
            cu.append(cu[-1] + k)
            req += [r_] * k
            slots.append(s)
        ids, req, cu, slots = ids + [0], req + [-1], cu + [cu[-1] + 1], slots + [0]  # (a row that belongs to no request)
        T = len(ids)
        stream = torch.full((T, hidden), 9.0, device=device())
        copy = torch.empty(T, hidden, dtype=td, device=device())
        K.embed_scaled(i32(ids), e.to(device()), stream, copy, last_tokens=last, token_req=i32(req), req_slots=i32(slots),
                       pairs=(b.to(device()), mp, mc, state, i32(cu)))
        K.raise_on_status()
        close(stream[:T - 1], torch.cat(want).float(), "float32", str(plan))
        assert torch.equal(copy, stream.to(td))
    for s in seqs:
        assert int(state[s]) == (seqs[s][at[s] - 1]) + 1
    assert not state[[1, 3]].any()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cols", [40, 37, 1024, 3000])
def test_outer_norms_and_plain_copies(dtype, cols):
    """The norm of a sum of two normed rows, and of the experts' weighted sum, on its way into the stream; the stream's rows
    as they are behind every kernel that can leave a next norm."""
    from ullm_b200.csrc import kernels

    K, T, td, eps = kernels(), 11, getattr(torch, dtype), 1e-3
    g = torch.Generator().manual_seed(cols)
    stream0 = torch.randn(T, cols, generator=g) * 2
    a, b = (torch.randn(T, cols, generator=g).to(td) for _ in range(2))
    wa, wb, wo = (1 + 0.3 * torch.randn(cols, generator=g) for _ in range(3))
    rms = lambda v: v.double() / torch.sqrt((v.double() ** 2).mean(-1, keepdim=True) + eps)
    dev = [t.to(device()) for t in (a, b, wa, wb, wo)]
    out = torch.empty(T, cols, dtype=td, device=device())
    both = 0.5 * (rms(a) * wa.double() + rms(b) * wb.double())
    for outer, ref in ((None, stream0.double() + both), ((dev[4], eps, 0.7), stream0.double() + 0.7 * rms(both) * wo.double())):
        s = stream0.to(device())
        K.pair_norm_add_norm(*dev[:4], eps, 0.5, stream=s, next_norm=(None, 0.0, 3, out), outer_norm=outer)
        close(s, ref.float(), "float32", f"pair, outer norm {outer is not None}")
        assert torch.equal(out, s.to(td))
    s = stream0.to(device())
    K.norm_scale_add(dev[0], s, dev[4], eps, 0.3, out)
    close(s, (stream0.double() + 0.3 * rms(a) * wo.double()).float(), "float32", "one normed operand")
    assert torch.equal(out, s.to(td))
    s = stream0.to(device())
    K.norm_add_norm(s, dev[0], dev[4], eps, 0.3, next_norm=(None, 0.0, 3, out))
    close(s, (stream0.double() + 0.3 * rms(a) * wo.double()).float(), "float32", "one normed operand, general kernel")
    assert torch.equal(out, s.to(td))
    rows = torch.randn(2 * T, cols, generator=g).to(td)
    place = torch.randperm(2 * T, generator=g).to(torch.int32)
    weight = torch.rand(T, 2, generator=g)
    y = (rows.double()[place.long()].view(T, 2, cols) * weight.double()[..., None]).sum(1)
    for outer, ref in ((None, stream0.double() + y), ((dev[4], eps), stream0.double() + rms(y) * wo.double())):
        s = stream0.to(device())
        assert K.moe_combine_add_norm(rows.to(device()), place.to(device()), weight.to(device()), 2, s,
                                      next_norm=(None, 0.0, 3, out), outer_norm=outer)
        close(s, ref.float(), "float32", f"experts, outer norm {outer is not None}")
        assert torch.equal(out, s.to(td))
    K.raise_on_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,mixes", [(64, 5), (50, 3), (256, 5)])
def test_token_shift_mixes(dtype, width, mixes):
    from ullm_b200.csrc import kernels

    K, td = kernels(), getattr(torch, dtype)
    g = torch.Generator().manual_seed(width)
    mu = torch.rand(mixes, width, generator=g)
    wide = torch.zeros(4, width + 12, device=device())
    state = wide[:, 8:8 + width]
    seqs = {s: torch.randn(12, width, generator=g).to(td) for s in (3, 0)}
    at = {3: 0, 0: 0}
    for plan in ([(3, 4), (0, 2)], [(0, 1), (3, 1)], [(3, 1)], [(3, 2), (0, 7)]):
        rows, cu, req, want = [], [0], [], []
        for i, (s, n) in enumerate(plan):
            x = seqs[s][:at[s] + n].double()
            m = x[None] + (pn.token_shift(x) - x)[None] * mu.double()[:, None, :]
            want.append(m[:, at[s]:])
            rows.append(seqs[s][at[s]:at[s] + n])
            at[s] += n
            cu.append(cu[-1] + n)
            req += [i] * n
        h = torch.cat(rows).to(device())
        out = torch.empty(mixes, h.shape[0], width, dtype=td, device=device())
        K.token_shift_mix(h, mu.to(device()), out, state, i32(cu), i32(req), i32([s for s, _ in plan]), len(plan),
                          single=all(n == 1 for _, n in plan))
        close(out.reshape(-1, width), torch.cat(want, 1).reshape(-1, width).float(), dtype, str(plan))
    K.raise_on_status()
    for s in seqs:
        assert torch.equal(state[s].cpu(), seqs[s][at[s] - 1].float())
    assert not wide[:, :8].any() and not wide[:, 8 + width:].any() and not wide[1:3].any()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,rank,n", [(3, 16, 64), (70, 5, 50), (33, 100, 200), (200, 64, 256), (1, 1, 1)])
def test_low_rank_decays(dtype, T, rank, n):
    from ullm_b200.csrc import kernels

    K, td = kernels(), getattr(torch, dtype)
    g = torch.Generator().manual_seed(T + rank)
    a = torch.randn(T, rank + 3, generator=g).to(td)
    w2 = (torch.randn(n, rank, generator=g) / rank ** 0.5).to(td)
    w0 = torch.randn(n, generator=g) * 2 - 3
    log = -torch.exp(torch.tanh(a[:, :rank].double()) @ w2.double().T + w0.double())
    out = torch.empty(T, n, device=device())
    av = a.to(device())[:, :rank]
    K.low_rank_decay(av, w2.to(device()), w0.to(device()), out)
    assert (out.cpu().double() - log.exp()).abs().max() < 2e-6
    K.low_rank_decay(av, w2.to(device()), w0.to(device()), out, log=True)
    assert ((out.cpu().double() - log) / log).abs().max() < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("G,T,rows,K_,extra", [(5, 3, 64, 128, 16), (5, 16, 96, 72, 8), (3, 8, 32, 512, 32), (4, 1, 64, 64, 0), (5, 40, 64, 64, 8), (3, 5, 20, 24, 8), (5, 7, 32, 64, 40), (5, 9, 32, 320, 200), (2, 30, 16, 40, 33)])
def test_products_with_an_operand_each(dtype, G, T, rows, K_, extra):
    from ullm_b200.csrc import kernels

    K, td = kernels(), getattr(torch, dtype)
    g = torch.Generator().manual_seed(G + T)
    N = (G - 1) * rows + extra if extra else G * rows
    x = torch.randn(G, T, K_, generator=g).to(td)
    w = (torch.randn(N, K_, generator=g) / K_ ** 0.5).to(td)
    out = torch.full((T, N), float("nan"), dtype=td, device=device())
    K.grouped_linear(x.to(device()), w.to(device()), out, rows)
    K.raise_on_status()
    ref = torch.cat([x[i].double() @ w[i * rows:(i + 1) * rows if i + 1 < G else N].double().T for i in range(G)], 1)
    close(out, ref.float(), dtype, "grouped products")


def _recurrence_batch(lens, slots, width, g):
    cu = [0]
    for k in lens:
        cu.append(cu[-1] + k)
    state = torch.randn(len(lens), width, generator=g) * 0.3
    return cu, i32(cu), i32(slots), i32([i for i, k in enumerate(lens) for _ in range(k)]), state


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dim", [(2, 64), (3, 20), (2, 7), (1, 128), (4, 32), (2, 48)])
def test_recurrence_with_a_bonus_against_the_plain_one(dtype, heads, dim):
    """Portions of unequal length in one batch, from states that are not zero, with decays from nearly one to nearly nothing:
    outputs and states of every form against 64-bit."""
    from ullm_b200.csrc import kernels
    from ullm_b200.engine.batch import Workspace

    K, td = kernels(), getattr(torch, dtype)
    lens, slots = (130, 5, 64, 1, 77), [4, 0, 1, 3, 2]
    g = torch.Generator().manual_seed(heads + dim)
    T, S = sum(lens), heads * dim
    qkv = (torch.randn(T, 3 * S + 8, generator=g) * 0.7).to(td)
    log = -torch.exp(torch.randn(T, S, generator=g) * 2 - 3)
    log[::17] = -60.0
    u = torch.randn(heads, dim, generator=g)
    cu, cu_q, req_slots, token_req, state0 = _recurrence_batch(lens, slots, heads * dim * dim + 8, g)
    ref = torch.zeros(T, heads, dim, dtype=torch.float64)
    ref_state = state0.double().clone()
    for i in range(len(lens)):
        S_ = state0[slots[i], :heads * dim * dim].double().view(heads, dim, dim).transpose(1, 2)  # [heads, key, value]
        for t in range(cu[i], cu[i + 1]):
            r, k, v = (qkv[t, o * S:(o + 1) * S].double().view(heads, dim) for o in range(3))
            kv = k[:, :, None] * v[:, None, :]
            ref[t] = torch.einsum("hkv,hk->hv", S_ + u.double()[:, :, None] * kv, r)
            S_ = log[t].double().exp().view(heads, dim, 1) * S_ + kv
        ref_state[slots[i], :heads * dim * dim] = S_.transpose(1, 2).reshape(-1)
    names = ["token by token"] + (["in chunks"] if K.gla_chunk_applies(td, heads, dim, dim) else [])
    assert len(names) == 1 + (dtype == "bfloat16" and dim % 16 == 0)
    qd, wd, ud = qkv.to(device()), log.exp().to(device()), u.to(device())
    for name in names:
        state, out = state0.to(device()), torch.full((T, S), float("nan"), device=device())
        most = 1 << 30
        if name == "in chunks":
            most = 16
            K.gla_chunk(qd, 0, S, 2 * S, wd, 1.0, K.gla_chunk_scratch(Workspace(device()), T, len(lens), heads, dim, dim), state,
                        cu_q, req_slots, token_req, out, len(lens), heads, dim, dim, 16, bonus=ud)
            assert torch.isnan(out[130:135]).all() and torch.isnan(out[199]).all() and not torch.isnan(out[:130]).any()
        K.gla_recurrence(qd, 0, S, 2 * S, wd.clone(), None, 0.0, 1.0, state, cu_q, req_slots, token_req, out, len(lens), heads,
                         dim, dim, bonus=ud, most_tokens=most)
        K.raise_on_status()
        close(out, ref.reshape(T, S).float(), "float32", f"{name}: outputs")
        close(state, ref_state.float(), "float32", f"{name}: states")


@pytest.mark.parametrize("heads,dim,vdim", [(2, 64, 32), (1, 128, 256), (3, 16, 48), (2, 96, 16), (1, 256, 64)])
def test_chunked_recurrence_without_a_bonus(heads, dim, vdim):
    """Queries with a factor, values of another width, the current token behind its own decay's step."""
    from ullm_b200.csrc import kernels
    from ullm_b200.engine.batch import Workspace

    K = kernels()
    lens, slots = (70, 17, 9, 128), [3, 1, 0, 2]
    g = torch.Generator().manual_seed(dim + vdim)
    T, S, V = sum(lens), heads * dim, heads * vdim
    qkv = (torch.randn(T, 2 * S + V + 8, generator=g) * 0.7).to(torch.bfloat16)
    w = torch.exp(-torch.exp(torch.randn(T, S, generator=g) * 2 - 3))
    w[::17] = 0.0
    cu, cu_q, req_slots, token_req, state0 = _recurrence_batch(lens, slots, heads * dim * vdim + 8, g)
    ref = torch.zeros(T, heads, vdim, dtype=torch.float64)
    ref_state = state0.double().clone()
    for i in range(len(lens)):
        S_ = state0[slots[i], :S * vdim].double().view(heads, vdim, dim)
        for t in range(cu[i], cu[i + 1]):
            q, k = (qkv[t, o * S:(o + 1) * S].double().view(heads, dim) for o in range(2))
            v = qkv[t, 2 * S:2 * S + V].double().view(heads, vdim)
            S_ = w[t].double().view(heads, 1, dim) * S_ + v[:, :, None] * k[:, None, :]
            ref[t] = torch.einsum("hvk,hk->hv", S_, q) * 0.3
        ref_state[slots[i], :S * vdim] = S_.reshape(-1)
    state, out = state0.to(device()), torch.full((T, V), float("nan"), device=device())
    qd, wd = qkv.to(device()), w.to(device())
    K.gla_chunk(qd, 0, S, 2 * S, wd, 0.3, K.gla_chunk_scratch(Workspace(device()), T, 4, heads, dim, vdim), state, cu_q, req_slots,
                token_req, out, 4, heads, dim, vdim, 16)
    K.gla_recurrence(qd, 0, S, 2 * S, wd.clone(), None, 0.0, 0.3, state, cu_q, req_slots, token_req, out, 4, heads, dim, vdim,
                     most_tokens=16)
    K.raise_on_status()
    close(out, ref.reshape(T, V).float(), "float32", "outputs")
    close(state, ref_state.float(), "float32", "states")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dim,vdim", [(2, 64, 48), (3, 32, 16), (2, 20, 13), (1, 128, 64)])
def test_fixed_decays_on_the_state_space_kernels(dtype, heads, dim, vdim):
    """One row of steps and decays for all tokens, a group per head, silu on the way in: token by token and in chunks."""
    from ullm_b200.csrc import kernels

    K, td = kernels(), getattr(torch, dtype)
    lens, slots = (100, 3, 64, 1), [2, 0, 3, 1]
    g = torch.Generator().manual_seed(dim)
    T, qk, vs = sum(lens), heads * dim, heads * vdim
    u = torch.randn(T, vs + 2 * qk + 8, generator=g).to(td)
    decay = torch.linspace(0.2, 0.9995, heads).double()
    cu, cu_q, req_slots, token_req, state0 = _recurrence_batch(lens, slots, heads * dim * vdim + 4, g)
    for fused in (True, False):
        x = pn.silu(u.double())
        if not fused:
            x = x.to(td).double()  # (the activation's kernel rounds)
        ref = torch.zeros(T, heads, vdim, dtype=torch.float64)
        ref_state = state0.double().clone()
        for i in range(len(lens)):
            S_ = state0[slots[i], :qk * vdim].double().view(heads, vdim, dim)
            for t in range(cu[i], cu[i + 1]):
                v, k, q = x[t, :vs].view(heads, vdim), x[t, vs:vs + qk].view(heads, dim), x[t, vs + qk:vs + 2 * qk].view(heads, dim)
                S_ = decay[:, None, None] * S_ + v[:, :, None] * k[:, None, :]
                ref[t] = torch.einsum("hvk,hk->hv", S_, q)
            ref_state[slots[i], :qk * vdim] = S_.reshape(-1)
        ud, state, out = u.to(device()), state0.to(device()), torch.empty(T, vs, device=device())
        ones, logs, zero = (t.float().to(device()) for t in (torch.ones(1, heads), decay.log()[None], torch.zeros(heads)))
        chunks = not fused and K.ssd_chunk_applies(td, heads, dim, vdim, heads)
        if not fused:
            K.act_rows("silu", ud[:, :vs + 2 * qk], ud[:, :vs + 2 * qk])
            assert torch.equal(ud[:, vs + 2 * qk:].cpu(), u[:, vs + 2 * qk:])
        if chunks:
            scores = torch.empty(K.ssd_chunk_floats(T, heads), device=device())
            K.ssd_chunk(ud, vs, vs + qk, ones, logs, zero, scores, state, cu_q, req_slots, token_req, out, len(lens), heads, dim,
                        vdim, heads, 16)
        K.ssd_recurrence(ud, vs, vs + qk, ones, logs, zero, state, cu_q, req_slots, token_req, out, len(lens), heads, dim, vdim,
                         heads, 16 if chunks else 1 << 30, silu_in=fused)
        K.raise_on_status()
        close(out, ref.reshape(T, vs).float(), "float32", f"outputs, silu on the way in {fused}", 1e-4 if fused else 3e-5)
        close(state, ref_state.float(), "float32", f"states, silu on the way in {fused}", 1e-4 if fused else 3e-5)
    # the norm over all heads with the gate behind it
    y, z, w = torch.randn(9, vs, generator=g), torch.randn(9, vs + 8, generator=g).to(td), 1 + 0.2 * torch.randn(vs, generator=g)
    got = torch.empty(9, vs, dtype=td, device=device())
    K.ssd_gate_norm(y.to(device()), z.to(device())[:, :vs], w.to(device()), 1, 1e-4, got, gate_behind=True)
    ref = pn.rms_norm(y.double(), w.double(), 1e-4) * torch.sigmoid(z[:, :vs].double())
    close(got, ref.float(), dtype, "gate behind the norm")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,n,cols,groups", [(2, 64, 64, 2), (4, 128, 64, 1), (3, 20, 13, 3), (2, 512, 24, 1), (1, 4, 1, 1), (6, 48, 80, 2), (2, 200, 40, 2)])
def test_single_tokens_through_a_state(dtype, heads, n, cols, groups):
    """Steps of one token per request, with a row that belongs to no request: state-space and per-channel decays, bonus and
    scale, silu on the way in, one row of decays for all tokens; other slots stay as they are."""
    from ullm_b200.csrc import kernels

    K, td = kernels(), getattr(torch, dtype)
    g = torch.Generator().manual_seed(n + cols)
    B, slots = 5, [3, 0, 5, 1, 2]
    T = B + 1
    sizes = heads * cols * n
    state0 = torch.randn(7, (sizes + 11) // 4 * 4, generator=g) * 0.5
    args = (i32(list(range(T + 1))), i32(slots + [0]), i32(list(range(B)) + [-1]))

    def check(name, out, state, ref, new):
        K.raise_on_status()
        assert not out[B].any()
        close(out[:B], ref.reshape(B, -1).float(), "float32", f"{name}: outputs")
        want = state0.clone().double()
        for b, s in enumerate(slots):
            want[s, :sizes] = new[b].reshape(-1)
        close(state, want.float(), "float32", f"{name}: states")

    # state-space form
    gs = groups * n
    xbc = torch.randn(T, heads * cols + 2 * gs + 3, generator=g).to(td)
    for one_row, silu in ((False, False), (True, True)):
        rows = 1 if one_row else T
        dt, logd, D = torch.rand(rows, heads, generator=g), -torch.rand(rows, heads, generator=g) * 3, torch.randn(heads, generator=g)
        x = pn.silu(xbc.double()) if silu else xbc.double()
        v = x[:B, :heads * cols].view(B, heads, cols)
        k, q = (x[:B, o:o + gs].view(B, groups, n).repeat_interleave(heads // groups, 1) for o in (heads * cols, heads * cols + gs))
        S = torch.stack([state0[s, :sizes].double().view(heads, cols, n) for s in slots])
        d = dt.double().expand(T, -1)[:B]
        new = logd.double().exp().expand(T, -1)[:B, :, None, None] * S + v[..., None] * (d[..., None] * k)[:, :, None, :]
        ref = torch.einsum("bhcn,bhn->bhc", new, q) + D.double()[None, :, None] * v
        state, out = state0.to(device()), torch.full((T, heads * cols), 5.0, device=device())
        K.ssd_recurrence(xbc.to(device()), heads * cols, heads * cols + gs, dt.to(device()), logd.to(device()), D.to(device()), state,
                         *args, out, T, heads, n, cols, groups, silu_in=silu, single=True)
        check(f"state space, one row {one_row}", out, state, ref, new)
    # a decay per key channel
    qkv = torch.randn(T, heads * (2 * n + cols) + 5, generator=g).to(td)
    q, k = (qkv[:B, o * heads * n:(o + 1) * heads * n].double().view(B, heads, n) for o in range(2))
    v = qkv[:B, 2 * heads * n:2 * heads * n + heads * cols].double().view(B, heads, cols)
    z, zb, u = torch.randn(T, heads * n, generator=g), torch.randn(heads * n, generator=g), torch.randn(heads, n, generator=g)
    for bonus in (False, True):
        w = torch.sigmoid(z.double()) if bonus else torch.sigmoid(z.double() + zb.double()) ** 0.25
        zin = w.float() if bonus else z
        w = w[:B].view(B, heads, 1, n)
        kv = v[..., None] * k[:, :, None, :]
        new = w * S + kv
        seen = S + u.double()[None, :, None, :] * kv if bonus else new
        ref = torch.einsum("bhcn,bhn->bhc", seen, q) * 0.6
        state, out = state0.to(device()), torch.full((T, heads * cols), 5.0, device=device())
        K.gla_recurrence(qkv.to(device()), 0, heads * n, 2 * heads * n, zin.to(device()), None if bonus else zb.to(device()),
                         0.0 if bonus else 0.25, 0.6, state, *args, out, T, heads, n, cols, bonus=u.to(device()) if bonus else None,
                         single=True)
        check(f"per-channel decays, bonus {bonus}", out, state, ref, new)


ATTENTION = [  # heads, kv heads, dim, vdim, pages of
    (4, 2, 64, 64, 16), (6, 1, 64, 80, 8), (2, 2, 128, 128, 16), (8, 1, 32, 48, 4), (16, 1, 128, 128, 16), (3, 3, 16, 96, 8),
    (4, 4, 20, 12, 8), (64, 1, 64, 64, 16)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv,dim,vdim,page", ATTENTION)
def test_attention_with_distance_biases_and_head_gates(dtype, heads, kv, dim, vdim, page):
    """The attention kernels alone on a mixed batch (portions, single tokens, a padding row) over shuffled pages: biases that
    are constant from distance 1, 40 and 150 on, a gate per head; with and without cutting the keys into runs."""
    from ullm_b200.csrc import kernels
    from ullm_b200.engine.batch import Workspace

    K, td = kernels(), getattr(torch, dtype)
    g = torch.Generator().manual_seed(heads * dim + page)
    held, new = (210, 64, 131, 7), (90, 1, 2, 7)
    B, T = len(held), sum(new) + 1
    per = -(-max(held) // page)
    pages = torch.randperm(B * per, generator=g).view(B, per)
    k = torch.randn(B * per * page, kv, dim, generator=g).to(td)
    v = torch.randn(B * per * page, kv, vdim, generator=g).to(td)
    q = (torch.randn(T, heads, dim, generator=g) * 1.5).to(td)
    gate = torch.randn(T, heads + 2, generator=g).to(td)
    scale = 0.7 / dim ** 0.5
    cu = [0]
    for n in new:
        cu.append(cu[-1] + n)
    table = pages.to(torch.int32).to(device())
    for length in (1, 40, 150):
        bias = torch.randn(heads, length, generator=g) * 2
        ref = torch.zeros(T, heads, vdim, dtype=torch.float64)
        for b in range(B):
            slots = (pages[b][:, None] * page + torch.arange(page)).reshape(-1)[:held[b]]
            kb, vb = (x.double()[slots].repeat_interleave(heads // kv, 1) for x in (k, v))
            for j in range(new[b]):
                i, t = held[b] - new[b] + j, cu[b] + j
                dist = (i - torch.arange(i + 1)).clamp(max=length - 1)
                s = torch.einsum("jhd,hd->hj", kb[:i + 1], q[t].double()) * scale + bias.double()[:, dist]
                ref[t] = torch.einsum("hj,jhv->hv", torch.softmax(s, -1), vb[:i + 1])
        gated = ref * torch.sigmoid(gate[:, :heads].double())[..., None]
        ws_ = Workspace(device())
        ctx = SimpleNamespace(decode_only=False, num_requests=B + 1, workspace=ws_)
        for use_gate, ws, step in ((False, None, None), (True, None, None), (True, ws_, None), (True, ws_, ctx), (False, ws_, ctx)):
            out = torch.full((T, heads * vdim), 7.0, dtype=td, device=device())
            K.pair_biased_rows = 1  # (short steps too)
            K.windowed_attention(q.view(T, -1).to(device()), out, k.view(-1, page, kv, dim).to(device()),
                                 v.view(-1, page, kv, vdim).to(device()), table, i32([0, 1, 2, 3, 0]), i32(cu + [T]),
                                 i32(list(held) + [0]), i32([b for b in range(B) for _ in range(new[b])] + [-1]), heads, kv, dim,
                                 vdim, page, 0, scale, gate=gate.to(device())[:, :heads] if use_gate else None,
                                 dist_bias=bias.to(device()), num_requests=B + 1, workspace=ws, ctx=step)
            K.raise_on_status()
            K.apply_switches(os.environ)
            path = "window_mma" if dtype == "bfloat16" and dim % 16 == 0 and vdim % 16 == 0 else "generic"
            if step is not None and dtype == "bfloat16" and dim == vdim == 128:
                path = "prefill_tcgen05"
            assert K.attention_path == path
            assert not out[T - 1].any()
            close(out[:T - 1], (gated if use_gate else ref)[:T - 1].reshape(T - 1, -1).float(), dtype,
                  f"biases to distance {length}, gate {use_gate}, runs {ws is not None}")


@pytest.mark.parametrize("heads,kv,dim,page", [(4, 2, 64, 16), (16, 1, 128, 8), (3, 3, 128, 16), (8, 4, 64, 4)])
def test_decode_attention_with_distance_biases_and_head_gates(heads, kv, dim, page):
    """Steps of single tokens on the split decode kernel, merged inside a cluster, by the second kernel, and unsplit."""
    from ullm_b200.csrc import kernels
    from ullm_b200.engine.batch import Workspace

    K = kernels()
    g = torch.Generator().manual_seed(heads + dim)
    held = (600, 1, 64, 257, 33)
    B, per = len(held), -(-max(held) // page)
    T = B + 1
    pages = torch.randperm(B * per, generator=g).view(B, per)
    k, v = (torch.randn(B * per * page, kv, dim, generator=g).to(torch.bfloat16) for _ in range(2))
    q = (torch.randn(T, heads, dim, generator=g) * 1.5).to(torch.bfloat16)
    gate = torch.randn(T, heads + 2, generator=g).to(torch.bfloat16)
    scale = 0.7 / dim ** 0.5
    ctx = SimpleNamespace(decode_only=True, num_requests=T, workspace=Workspace(device()))
    for length in (1, 40, 300):
        bias = torch.randn(heads, length, generator=g) * 2
        ref = torch.zeros(B, heads, dim, dtype=torch.float64)
        for b in range(B):
            slots = (pages[b][:, None] * page + torch.arange(page)).reshape(-1)[:held[b]]
            kb, vb = (x.double()[slots].repeat_interleave(heads // kv, 1) for x in (k, v))
            dist = (held[b] - 1 - torch.arange(held[b])).clamp(max=length - 1)
            s = torch.einsum("jhd,hd->hj", kb, q[b].double()) * scale + bias.double()[:, dist]
            ref[b] = torch.einsum("hj,jhv->hv", torch.softmax(s, -1), vb)
        for merge in (True, False, "one"):
            K.decode_cluster_merge, K.decode_split_target = (merge, 400) if merge != "one" else (False, 1)
            for use_gate in (True, False):
                out = torch.full((T, heads * dim), 7.0, dtype=torch.bfloat16, device=device())
                K.windowed_attention(q.view(T, -1).to(device()), out, k.view(-1, page, kv, dim).to(device()),
                                     v.view(-1, page, kv, dim).to(device()), pages.to(torch.int32).to(device()),
                                     i32([0, 1, 2, 3, 4, 0]), i32(list(range(T + 1))), i32(list(held) + [0]), i32([0, 1, 2, 3, 4, -1]),
                                     heads, kv, dim, dim, page, 0, scale, gate=gate.to(device())[:, :heads] if use_gate else None,
                                     dist_bias=bias.to(device()), num_requests=T, workspace=ctx.workspace, ctx=ctx)
                K.raise_on_status()
                assert K.attention_path == "decode" and not out[B].any()
                want = ref * torch.sigmoid(gate[:B, :heads].double())[..., None] if use_gate else ref
                close(out[:B], want.reshape(B, -1).float(), "bfloat16", f"biases to distance {length}, merge {merge}, gate {use_gate}")
            K.apply_switches(os.environ)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_biases_weights_and_scales_each_show(tmp_path, dtype):
    """A model whose biases, gates, norms, temperature and scales are far from what leaves them unseen: portions against the
    plain model, and the plain model itself changes when one is left out."""
    cfg = config(56, 80, [parallel(left(4, 2, 16, 24, 0.25, 3, 12, coef=1.5, every=6), right(4, 8, 12, 2, 4, 2), moe(4, 2, 24)),
                          wkv(2, 16, dense(32)), lightning(16, 16, [0.95, 0.6], moe(3, 1, 24))], logit_scale=0.2)
    w = pn.random_weights(cfg, seed=33)
    for n in "qkv":
        w[f"l0.mix.left.{n}.b"] = w[f"l0.mix.left.{n}.b"] * 4
    w["l0.mix.left.g"] = w["l0.mix.left.g"] * 3
    w["l0.mix.left.rel"] = w["l0.mix.left.rel"] * 2
    w["l0.mix.right.D"] = torch.tensor([2.0, -1.0, 0.5, 3.0])
    w["l0.mix.left.out"], w["l0.mix.right.out"] = torch.linspace(0.2, 2.0, 56), torch.linspace(2.0, 0.2, 56)
    w["l1.norm1"], w["l1.norm2"] = torch.linspace(-0.9, 1.0, 56), torch.linspace(1.0, -0.9, 56)
    w["l1.mix.u"] = w["l1.mix.u"] * 8
    w = cast({n: t.to(torch.bfloat16).float() for n, t in w.items()}, dtype)
    cfg = cfg if dtype == "float32" else every_expert_chosen(cfg)
    ids = random_ids(80, 40, 2)
    ref = oracle(ids, w, cfg)

    def off(w2=None, cfg2=None):
        return float((oracle(ids, w2 or w, cfg2 or cfg) - ref).abs().max() / ref.abs().max())

    names = ["bigram", "l0.mix.left.v.b", "l0.mix.left.rel", "l0.mix.left.g", "l0.mix.right.D", "l1.mix.u", "l1.norm1", "l1.norm2",
             "final.norm", "l1.mix.mu.k"] + (["l0.mix.left.q.b", "l0.mix.left.k.b", "l1.mix.w1", "l1.mix.mu.w"] if dtype == "float32" else [])
    for name in names:
        assert off({**w, name: torch.zeros_like(w[name])}) > 3 * TOL[dtype], name
    for name in ("l0.mix.left.out", "l0.mix.right.out", "l0.mix.left.q.norm", "l1.mix.norm") + (("l2.mix.norm",) if dtype == "float32" else ()):
        assert off({**w, name: torch.ones_like(w[name])}) > 3 * TOL[dtype], name
    other = copy.deepcopy(cfg)
    other["layers"][0]["mixer"]["left"]["q_temp"]["coef"] = 0.0
    assert off(cfg2=other) > 2 * TOL[dtype], "temperature"
    r = make_runner(tmp_path, cfg, w, 8, dtype)
    got = replay(r, {"a": ids}, [[("a", 17)], [("a", 2)], [("a", 21)]])["a"]
    assert_rows_close(got, ref, dtype, "biases, norms, gates and scales")


# ---------------------------------------------------------------------------------------------------------
# whole prompts, token-by-token decoding, portions
# ---------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["A", "B", "C", "D", "E", "F"])
def test_whole_decode_and_portions_agree_with_the_plain_model(tmp_path, dtype, tag):
    if tag == "D" and dtype != "float32":
        pytest.skip("heads of one number have only a sign behind their norm: 16-bit rounding flips it")
    cfg, w, page = model_for(tag, dtype)
    r = make_runner(tmp_path, cfg, w, page, dtype, num_pages=64)
    n = 75 if tag not in ("E", "F") else 190
    ids = random_ids(cfg["vocab"], n, 11)
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
        assert_model_close(got, ids, w, cfg, dtype, f"{tag} {name}")


@pytest.mark.parametrize("tag,dtype", [("A", "float32"), ("F", "float32"), ("E", "float32"), ("E", "bfloat16")])
def test_unequal_batches_with_pages_and_slots_used_again(tmp_path, dtype, tag):
    """Three request slots and a pool that cannot hold all requests at once: six requests of unequal length come
    and go, portions of some beside single tokens of others; every request equals itself run alone."""
    cfg, w, page = model_for(tag, dtype)
    pages = 24 if tag == "A" else 14  # (fewer than all requests together hold)
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
        assert_model_close(got[k], reqs[k], w, cfg, dtype, f"request {k}")
    assert not r.cache.requests
    assert all(r.cache.num_free_pages(g) == n for g, n in enumerate(r.cache.group_pages))


# ---------------------------------------------------------------------------------------------------------
# distances: bucket edges, far keys, page borders; weights made so that one key or one bucket decides
# ---------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,most,bucket,dim,vdim", [
    (10, 40, 4, 16, 16), (10, 40, 5, 64, 64), (10, 40, 7, 32, 48), (12, 300, 10, 128, 128), (12, 300, 11, 64, 64), (8, 30, 0, 24, 20),
    (16, 128, 12, 64, 80), (5, 90, 3, 128, 128)])
def test_bucket_edges_in_prompts_and_decoding(tmp_path, dtype, rows, most, bucket, dim, vdim):
    """One row of the distance table is far above the others, so a query sees almost nothing but the keys at the bucket's
    distances: a key at a wrong side of an edge changes the logits by much more than any tolerance."""
    cfg = config(48, 61, [parallel(left(2, 1, dim, vdim, 0.5 / dim ** 0.5, 1, most), right(2, 8, 8, 1, 2, 1))])
    w = pn.random_weights(cfg, seed=rows + bucket, bias_rows=rows)
    w["l0.mix.left.rel"] = torch.full((rows, 2), -4.0)
    w["l0.mix.left.rel"][bucket] = 8.0
    w["l0.mix.right.out"] = w["l0.mix.right.out"] * 0.25
    w = cast(w, dtype)
    buckets = [pn.distance_bucket(i, rows, most) for i in range(400)]
    first = buckets.index(bucket)
    n = first + 60
    ids = random_ids(61, n, 3)
    ref = oracle(ids, w, cfg)
    keep = pn.distance_bucket
    offs = []
    for shift in (1, -1):  # the test has power: edges one distance farther or nearer are far off
        pn.distance_bucket = lambda i, r_, m_, s=shift: keep(max(0, i + s), r_, m_)
        try:
            offs.append(float((oracle(ids, w, cfg) - ref).abs().max() / ref.abs().max()))
        finally:
            pn.distance_bucket = keep
    assert min(offs) > 5 * TOL[dtype], offs
    r = make_runner(tmp_path, cfg, w, 8, dtype, num_pages=60)
    cuts = [7, 1, 1, 8, 2, first] if first > 1 else [7, 1, 1, 8, 2]
    plan = [[("a", k)] for k in cuts] + [[("a", 1)] for _ in range(n - sum(cuts))]
    for name, got in (("cut", replay(r, {"a": ids}, plan)["a"]), ("whole", replay(r, {"b": ids}, [[("b", n)]])["b"])):
        if dtype == "float32":
            assert_close(got, ref, dtype, name)
        else:
            mx, _ = errors(got, ref)
            assert mx <= max(TOL[dtype], min(offs) / 4), f"{name}: {mx:.3e} of scale (a wrong edge: {min(offs):.3e})"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,vdim", [(24, 20), (64, 112), (128, 128)])
def test_a_far_key_among_hundreds_decides(tmp_path, dtype, dim, vdim):
    """At the end of 400 tokens the asking token's query matches the key of ONE marked token near the start, and the logits
    say which token stood there (a rank-one W_q on its embedding)."""
    H = 2
    cfg = config(48, 61, [parallel(left(H, 1, dim, vdim, 1.0 / dim, 2, 30, coef=0.0), right(2, 8, 8, 1, 2, 1))])
    w = pn.random_weights(cfg, seed=dim)
    asks, marked, other = 58, 60, 59
    w["bigram"] = torch.zeros_like(w["bigram"])
    for n in "qkv":
        w[f"l0.mix.left.{n}.b"] = torch.zeros_like(w[f"l0.mix.left.{n}.b"])
        w[f"l0.mix.left.{n}.conv"] = torch.zeros_like(w[f"l0.mix.left.{n}.conv"])
        w[f"l0.mix.left.{n}.conv"][:, -1] = 1.0
    w["l0.mix.left.k.norm"] = torch.ones(dim)
    w["l0.mix.left.q.norm"] = torch.full((dim,), 32.0)
    key = w["l0.mix.left.k"].double() @ w["embed"][marked].double()
    wq = key[:, None] * w["embed"][asks].double()[None, :] / float(w["embed"][asks].double().pow(2).sum())
    w["l0.mix.left.q"] = wq.repeat(H, 1).to(torch.bfloat16).float()
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
    whole = replay(r, {"b": ids}, [[("b", n)]])["b"]
    for g in (got, whole):
        assert_close(g[-1:], ref[-1:], dtype, "far key, last row")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layer", [wkv(2, 12), wkv(2, 64), wkv(1, 32), lightning(20, 12, [0.9999, 1.0]), lightning(64, 64, [0.9998, 0.9999])],
                         ids=["wkv12", "wkv64", "wkv32", "lin20", "lin64"])
def test_states_remember_one_token_over_portions_and_single_tokens(tmp_path, dtype, layer):
    """Decays of nearly one, and only two tokens of the vocabulary write to the state at all (their keys read two channels
    that every other token has at zero): which of them stood 260 positions back shows in the last logits.  A lost, doubled or
    mixed-up state would be far off."""
    cfg = config(48, 61, [layer])
    w = pn.random_weights(cfg, seed=9)
    marked, other = 60, 59
    w["bigram"] = torch.zeros_like(w["bigram"])
    e = w["embed"]
    e[:, :2], e[:, 2] = 0.0, 1.0
    e[marked, 0], e[other, 1] = 4.0, 4.0
    m, q = "l0.mix.", "r" if layer["type"] == "wkv" else "q"
    k_row = w[m + "k"][:, :2].abs().mean(1) + 0.5
    w[m + "k"] = torch.zeros_like(w[m + "k"])
    w[m + "k"][:, 0] = w[m + "k"][:, 1] = k_row  # (positive keys for the two tokens, zero for all others)
    w[m + q] = torch.zeros_like(w[m + q])
    w[m + q][:, 2] = 1.0  # (every token asks alike)
    w[m + "v"] = w[m + "v"] * 3
    if layer["type"] == "wkv":
        for s in "rkv":
            w[m + "mu." + s] = torch.zeros(48)
        w[m + "w0"] = torch.full_like(w[m + "w0"], -9.5)
        w[m + "w2"] = w[m + "w2"] * 0.1
    w = cast({n: t.to(torch.bfloat16).float() for n, t in w.items()}, dtype)
    n = 290
    ids = [t % 58 for t in random_ids(61, n, 3)]
    ids[30] = marked
    ref = oracle(ids, w, cfg)
    changed = list(ids)
    changed[30] = other
    assert (oracle(changed, w, cfg)[-1] - ref[-1]).abs().max() > 3 * TOL[dtype] * ref.abs().max(), "token 30 must matter at the end"
    r = make_runner(tmp_path, cfg, w, 8, dtype, num_pages=56)
    for name, plan in (("portions", [64, 2, 2, 100, 2, 64, 1, 3, 2]), ("decode", [40]), ("whole", [n])):
        plan = [[(name, k)] for k in plan]
        plan += [[(name, 1)] for _ in range(n - sum(k for (_, k), in plan))]
        got = replay(r, {name: ids}, plan)[name]
        assert_close(got[-1:], ref[-1:], dtype, f"memory, {name}, last row")
        assert_rows_close(got, ref, dtype, f"memory, {name}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_first_tokens_alone_and_in_pairs(tmp_path, dtype):
    """Requests of one, two and three tokens, each alone in a step and side by side: the last row of the pair table, no row
    before the first, a softmax over one key, convolutions over zeros, empty states."""
    for tag in ("A", "B", "C"):
        cfg, w, page = model_for(tag, dtype)
        r = make_runner(tmp_path, cfg, w, page, dtype, name=tag)
        reqs = {k: random_ids(cfg["vocab"], n, 7 + n) for k, n in dict(a=1, b=2, c=3, d=2).items()}
        got = replay(r, reqs, [[("a", 1)], [("b", 2), ("c", 1)], [("c", 2), ("d", 1)], [("d", 1)]])
        for k in reqs:
            assert_model_close(got[k], reqs[k], w, cfg, dtype, f"{tag} request {k}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(tmp_path, dtype):
    """One prompt token, then 300 tokens one by one: every state is carried 300 times, pages are added."""
    cfg, w, page = model_for("B", dtype)
    r = make_runner(tmp_path, cfg, w, page, dtype, num_pages=160)
    ids = random_ids(cfg["vocab"], 301, 17)
    got = replay(r, {"a": ids}, [[("a", 1)] for _ in range(301)])["a"]
    assert_model_close(got, ids, w, cfg, dtype, "long decoding")


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
    compared = 0
    for p, o in zip(prompts, outs):
        assert len(o.token_ids) == 14
        seq = list(p)
        for tok in o.token_ids:
            lg = pn.forward(cfg, wd, seq)[-1]
            top2 = torch.topk(lg, 2).values
            if top2[0] - top2[1] > 1e-3 * lg.abs().max():
                assert tok == int(torch.argmax(lg)), f"prompt of {len(p)}: token {len(seq) - len(p)} differs"
                compared += 1
            seq.append(tok)
    assert compared > 50
    llm.engine.runner.cache.check_invariants()
