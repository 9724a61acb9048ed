"""Host-side pieces of the Mafarax decoder that need no GPU: the config.json reader, the tensor names the model declares,
what the cache manager plans for and gives back from stretches of positions, and the plain implementation's own reading
of each mechanism."""

import copy
import json

import pytest
import torch

import plain_mafarax as pm
from mafarax_helpers import CFG_A, CFG_B, CFG_C, CFG_D, CFG_E

ALL = (CFG_A, CFG_B, CFG_C, CFG_D, CFG_E)


def _model(cfg):
    from ullm_b200.config import load_model_spec
    from ullm_b200.parts.model import DecoderModel

    return DecoderModel(load_model_spec(copy.deepcopy(cfg))[1])


def _shapes(cfg):
    return {n: tuple(s) for n, (s, _) in pm.tensor_shapes(cfg).items()}


def test_the_model_declares_exactly_the_checkpoints_tensors():
    for cfg in ALL:
        model = _model(cfg)
        assert {n: tuple(d.shape) for n, d in model.all_decls().items()} == _shapes(cfg)
        assert model.spec.stream_dtype == "float32" and not model.spec.tie_embeddings
        assert model.spec.logit_scale == cfg["logit_scale"]


def test_allocated_tensors_have_the_declared_names_and_32_bit_where_the_arithmetic_is():
    for cfg in (CFG_A, CFG_C):
        model = _model(cfg)
        model.allocate("cpu", torch.bfloat16)
        t = model.all_tensors()
        assert {n: tuple(v.shape) for n, v in t.items()} == _shapes(cfg)
        for n, v in t.items():
            is32 = ("norm" in n or n.endswith((".out", ".conv.b", ".dt_bias", ".A_log", ".D")))
            assert v.dtype == (torch.float32 if is32 else torch.bfloat16), n


def test_both_sides_share_one_input_product_and_a_shared_expert_of_equal_size_the_experts_stack():
    model = _model(CFG_A)
    model.allocate("cpu", torch.float32)
    for i, b in enumerate(model.blocks):
        mix = b.mixer
        q, into = (model.all_tensors()[f"l{i}.mix.{n}"] for n in ("left.q", "right.in"))
        assert q.data_ptr() == mix.w_in.data_ptr()
        assert into.data_ptr() == mix.w_in[mix.left_cols].data_ptr() and mix.left_cols % 8 == 0
        used = mix.left.input_width()
        assert not mix.w_in[used:mix.left_cols].any() and not mix.b_in[used:].any()
    first, last = model.blocks[0].feed_forward, model.blocks[2].feed_forward
    assert not first.rides and last.rides
    assert model.all_tensors()["l2.mlp.shared.up"].data_ptr() == last.w_gate_up[8].data_ptr()
    assert first.w_gate_up.shape == (6, 48, 72) and last.w_down.shape == (9, 72, 32)


@pytest.mark.parametrize("change,needle", [
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["norm"].update(eps=0), "eps"),
    (lambda c: c.update(logit_scale="1"), "logit_scale"),
    (lambda c: c["layers"][0].update(type="attention"), "type"),
    (lambda c: c["layers"][0].pop("mixer"), "mixer"),
    (lambda c: c["layers"][0]["mixer"].pop("left"), "heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=26), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(base=-1), "base"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=0), "factor"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("state"), "state"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(groups=3), "groups"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "groups"),
    (lambda c: c["layers"][0]["mlp"]["shared"].pop("ff"), "ff"),
])
def test_config_errors_name_the_key(change, needle):
    from ullm_b200.config import load_model_spec
    from ullm_b200.config.mafarax import MafaraxConfigError

    cfg = copy.deepcopy(CFG_A)
    change(cfg)
    with pytest.raises(MafaraxConfigError, match=needle):
        load_model_spec(cfg)


def test_random_model_folder_round_trip(tmp_path):
    from ullm_b200.config import load_model_spec
    from ullm_b200.engine.cli import main
    from ullm_b200.weights.safetensors_io import open_model_files

    path = tmp_path / "cfg.json"
    path.write_text(json.dumps(CFG_B))
    out = str(tmp_path / "model")
    assert main(["random-model", "--out", out, "--config", str(path), "--seed", "3", "--dtype", "bfloat16"]) == 0
    files = open_model_files(out)
    shapes = {n: tuple(f.shape(n)) for f in files for n in f.names()}
    for f in files:
        f.close()
    assert shapes == _shapes(CFG_B)
    cfg, spec = load_model_spec(out)
    assert spec.architecture == "Mafarax" and cfg.to_dict()["layers"] == CFG_B["layers"]


def test_stretches_form_groups_by_size_and_each_layer_has_pages_and_a_state_row():
    from ullm_b200.cache.manager import plan_groups_with_aux

    needs = _model(CFG_A).cache_needs()
    groups, where, aux = plan_groups_with_aux(needs)
    assert [g.need.chunk for g in groups] == [9, 20, 13] and all(g.need.window is None for g in groups)
    assert all(w is not None for w in where) and all(a is None for a in aux)
    assert (needs[0][0].num_kv_heads, needs[0][0].head_dim, needs[0][0].v_dim) == (2, 24, 40)
    # S of every head, then the last taps - 1 rows of x | B | C
    assert needs[0][1].shape == (4 * 12 * 20 + 3 * (4 * 12 + 2 * 2 * 20),) and needs[0][1].dtype == torch.float32
    d = _model(CFG_D).cache_needs()
    assert d[1][0].keeps_all and d[0][0].chunk == 1 and d[0][1].shape == (16,)  # one tap: no rows to remember


@pytest.mark.parametrize("size,page", [(8, 4), (9, 4), (5, 4), (4, 4), (1, 4), (3, 4), (7, 2)])
def test_pages_of_a_finished_stretch_go_back_at_its_edge(size, page):
    """Token by token and in portions: after every step exactly the pages that hold positions of the next token's own
    stretch (or beyond) are held; a page whose last position lies before it is free."""
    from ullm_b200.cache import CacheManager
    from ullm_b200.parts import CacheNeed

    for steps in ([1] * 40, [2] * 20, [7, 1, 11, 1, 1, 19], [40]):
        m = CacheManager([(CacheNeed(1, 8, chunk=size), None, None)], page, 20, 2, 20, device=None)
        rc = m.admit("a")
        n = 0
        for k in steps:
            m.reserve(rc, k)
            slots = [int(s) for s in m.slot_mapping(rc, 0, k)]
            assert len(set(slots)) == k and min(slots) >= 0
            m.commit(rc, k)
            n += k
            start = n - n % size  # where the next token's stretch begins
            held = {i for i, p in enumerate(rc.pages[0]) if p >= 0}
            assert held == {i for i in range(-(-n // page)) if (i + 1) * page > start}, (n, held)
            m.check_invariants()
        m.release(rc)
        assert m.num_free_pages() == 20
        assert m.tree is None  # no prefix reuse: a later request could not see what was given back


def test_a_reader_of_another_layers_cache_keeps_what_both_can_see():
    from ullm_b200.cache import plan_groups
    from ullm_b200.parts import CacheNeed

    c8, c5, w6, full = CacheNeed(1, 8, chunk=8), CacheNeed(1, 8, chunk=5), CacheNeed(1, 8, 6), CacheNeed(1, 8)

    def kept(writer, reader):
        groups, where = plan_groups([(writer, None, None), (reader, None, 0)])
        assert where == [(0, 0), (0, 0)]
        return groups[0].need

    assert kept(c8, c8).chunk == 8
    assert (kept(c8, c5).window, kept(c8, c5).chunk) == (8, None)  # a window of 8 holds both kinds of stretches
    assert kept(c5, w6).window == 6 and kept(w6, c8).window == 8
    assert kept(c8, full).keeps_all and kept(full, c8).keeps_all


# ---------------------------------------------------------------------------------------------------------
# the plain implementation's own reading of each mechanism, against direct evaluations
# ---------------------------------------------------------------------------------------------------------
def test_plain_stretches_see_their_own_positions_only():
    g = torch.Generator().manual_seed(4)
    q, k, v = (torch.randn(2, 9, 4, generator=g).double() for _ in range(3))
    out = pm.chunked_attention_core(q, k[:1], v[:1], 0.5, 4).reshape(9, 2, 4)
    for i, lo in ((0, 0), (3, 0), (4, 4), (7, 4), (8, 8)):
        for h in range(2):
            p = torch.softmax(k[0, lo:i + 1] @ q[h, i] * 0.5, 0)
            assert torch.allclose(out[i, h], p @ v[0, lo:i + 1], rtol=1e-10, atol=1e-12)
    assert torch.allclose(out[4], v[0, 4].expand(2, 4)) and torch.allclose(out[8], v[0, 8].expand(2, 4))


def test_plain_rotation_divides_the_frequencies():
    v = torch.randn(3, 10, generator=torch.Generator().manual_seed(2)).double()
    pos = torch.tensor([0, 5, 11])
    b = pm.rotate_halves(v, pos, 6, 100.0, 4.0)
    for t, p in enumerate(pos.tolist()):
        for i in range(3):
            ang = torch.tensor(p * 100.0 ** (-2.0 * i / 6) / 4.0).double()
            assert torch.allclose(b[t, i], v[t, i] * torch.cos(ang) - v[t, i + 3] * torch.sin(ang))
            assert torch.allclose(b[t, i + 3], v[t, i + 3] * torch.cos(ang) + v[t, i] * torch.sin(ang))
    assert torch.equal(b[:, 6:], v[:, 6:])
    from ullm_b200.parts.position import scaled_frequencies

    f = scaled_frequencies(6, 100.0, dict(factor=4.0))
    assert torch.allclose(f, torch.tensor([100.0 ** (-2.0 * i / 6) / 4.0 for i in range(3)]).double(), rtol=1e-14)


def test_plain_recurrence_equals_the_sum_over_decayed_pairs():
    """y_t = sum_s exp(-exp(A) sum_{s<u<=t} dt_u) dt_s (C_t . B_s) x_s + D x_t."""
    g = torch.Generator().manual_seed(3)
    n, H, P, G, N = 11, 4, 3, 2, 5
    x, B, C = torch.randn(n, H, P, generator=g).double(), torch.randn(n, G, N, generator=g).double(), torch.randn(n, G, N, generator=g).double()
    dt = torch.rand(n, H, generator=g).double()
    a_log, D = torch.randn(H, generator=g).double(), torch.randn(H, generator=g).double()
    y = pm.state_space_core(x, B, C, dt, a_log, D)
    for h in range(H):
        for t in (0, 4, n - 1):
            ref = D[h] * x[t, h]
            for s in range(t + 1):
                ref = ref + torch.exp(-torch.exp(a_log[h]) * dt[s + 1:t + 1, h].sum()) * dt[s, h] * (C[t, h // 2] @ B[s, h // 2]) * x[s, h]
            assert torch.allclose(y[t, h], ref, rtol=1e-10, atol=1e-12)


def test_plain_convolution_reads_only_the_past_and_adds_the_bias():
    u = torch.arange(12.0).view(6, 2).double()
    w = torch.tensor([[1.0, 10.0, 100.0], [0.0, 0.0, 1.0]]).double()
    silu = lambda z: z * torch.sigmoid(z)
    y = pm.causal_conv_silu(u, w, torch.tensor([3.0, -1.0]).double())
    assert torch.allclose(y[:, 1], silu(u[:, 1] - 1.0))
    assert torch.allclose(y[0, 0], silu(100 * u[0, 0] + 3)) and torch.allclose(y[2, 0], silu(u[0, 0] + 10 * u[1, 0] + 100 * u[2, 0] + 3))


def test_plain_choice_goes_by_groups_and_the_weight_by_the_score():
    w = {"router": torch.eye(6).double()}
    h = torch.tensor([[5.0, -5.0, 1.0, 1.1, 2.0, -1.0]]).double()  # groups (0 1) (2 3) (4 5)
    s = torch.sigmoid(h[0])
    chosen, weight = pm.route(h, w, "", dict(experts=6, top=2, scale=3.0, groups=dict(count=3, keep=1)))
    assert chosen.tolist() == [[3, 2]]  # the largest score of all lies in a group that is not kept
    assert torch.allclose(weight[0], 3.0 * s[[3, 2]])
    chosen, _ = pm.route(h, w, "", dict(experts=6, top=2, scale=1.0, groups=dict(count=3, keep=2)))
    assert chosen.tolist() == [[4, 3]]
    chosen, _ = pm.route(h, w, "", dict(experts=6, top=2, scale=1.0))
    assert chosen.tolist() == [[0, 4]]


def test_plain_gate_comes_before_the_norm_and_each_part_has_its_own():
    g = torch.Generator().manual_seed(6)
    y, z, w = torch.randn(3, 6, generator=g).double(), torch.randn(3, 6, generator=g).double(), torch.randn(6, generator=g).double()
    out = pm.gate_then_group_norm(y, z, 2, w, 1e-3)
    v = y * z * torch.sigmoid(z)
    for a in (0, 3):
        p = v[:, a:a + 3]
        assert torch.allclose(out[:, a:a + 3], p / torch.sqrt((p ** 2).mean(-1, keepdim=True) + 1e-3) * w[a:a + 3])
