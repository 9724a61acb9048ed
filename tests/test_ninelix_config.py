"""Host-side pieces of the Ninelix decoder that need no GPU: the config.json reader, sizes that only tensors give, the
tensor names the model declares, what the cache manager plans, and the plain implementation's own reading of each mechanism."""

import copy
import json
import math

import pytest
import torch

import plain_ninelix as pn
from ninelix_helpers import (CFG_A, CFG_B, CFG_C, CFG_E, CONFIGS, TENSOR_SIZES, config, dense, left, lightning, oracle, parallel,
                             right, weights_for, wkv, write_model)


def _shapes(tag):
    return {n: tuple(s) for n, (s, _) in pn.tensor_shapes(CONFIGS[tag][0], **TENSOR_SIZES[tag]).items()}


def _model(tag):
    from ullm_b200.config.ninelix import NinelixConfig, ninelix_model_spec
    from ullm_b200.parts.model import DecoderModel

    return DecoderModel(ninelix_model_spec(NinelixConfig.from_dict(copy.deepcopy(CONFIGS[tag][0]), _shapes(tag))))


def test_the_model_declares_exactly_the_checkpoints_tensors():
    for tag, (cfg, _) in CONFIGS.items():
        model = _model(tag)
        assert {n: tuple(d.shape) for n, d in model.all_decls().items()} == _shapes(tag)
        assert model.spec.stream_dtype == "float32" and not model.spec.tie_embeddings
        assert model.spec.logit_scale == cfg["logit_scale"]


def test_allocated_tensors_have_the_declared_names_and_32_bit_where_the_arithmetic_is():
    for tag in ("A", "C"):
        model = _model(tag)
        model.allocate("cpu", torch.bfloat16)
        t = model.all_tensors()
        assert {n: tuple(v.shape) for n, v in t.items()} == _shapes(tag)
        for n, v in t.items():
            is32 = "norm" in n or ".mu." in n or n.endswith((".out", ".conv.b", ".dt_bias", ".A_log", ".D", ".rel", ".w0", ".u"))
            assert v.dtype == (torch.float32 if is32 else torch.bfloat16), n


def test_stacked_products_share_memory_with_the_checkpoints_tensors():
    model = _model("A")
    model.allocate("cpu", torch.float32)
    t = model.all_tensors()
    par, tm, lin = (model.blocks[i].mixer for i in (0, 1, 2))
    assert t["l0.mix.left.g"].data_ptr() == par.w_in[par.left.qkv_rows].data_ptr() and par.left.w_rows == par.left.qkv_rows + 4
    assert t["l0.mix.right.in"].data_ptr() == par.w_in[par.left_cols].data_ptr() and par.left_cols % 8 == 0
    assert not par.b_in[par.left.qkv_rows:].any()  # the gate has no bias
    assert t["l1.mix.w1"].data_ptr() == tm.w_in[4 * tm.size].data_ptr() and t["l1.mix.mu.k"].data_ptr() == tm.mu[1].data_ptr()
    assert t["l2.mix.v"].data_ptr() == lin.w_in.data_ptr() and t["l2.mix.q"].data_ptr() == lin.w_in[lin.v_size + lin.qk_size].data_ptr()


def test_derived_values_are_formed_when_the_weights_are_there(tmp_path):
    from ullm_b200.config import load_model_spec
    from ullm_b200.parts.model import DecoderModel
    from ullm_b200.weights import load_weights

    cfg, w, _ = weights_for("A", "float32")
    d = write_model(str(tmp_path / "m"), cfg, w)
    model = DecoderModel(load_model_spec(d)[1])
    model.allocate("cpu", torch.float32)
    with pytest.raises(RuntimeError, match="loaded"):
        model.final_norm.weight
    load_weights(model, d)
    assert torch.equal(model.final_norm.weight, 1.0 + w["final.norm"])
    assert torch.equal(model.blocks[1].mixer_norm.rms_params()[0], 1.0 + w["l1.norm1"])
    a = model.blocks[0].mixer.left
    for n in (0, 1, 4, 5, 19, 20, 500):
        row = a.bias_table[:, min(n, a.bias_table.shape[1] - 1)]
        assert torch.equal(row, w["l0.mix.left.rel"][pn.distance_bucket(n, 10, 20)]), n


@pytest.mark.parametrize("rows,most", [(2, 2), (2, 50), (3, 7), (4, 14), (6, 9), (9, 33), (10, 20), (16, 128), (16, 2000), (32, 60), (32, 512), (31, 1000)])
def test_distance_buckets(rows, most):
    from ullm_b200.parts.position import distance_buckets

    got = distance_buckets(rows, most)
    assert got == [pn.distance_bucket(n, rows, most) for n in range(len(got))]
    assert got[:rows // 2] == list(range(rows // 2)) and got == sorted(got)
    assert got[-1] == rows - 1 and rows - 1 not in got[:-1] and len(got) <= most + 1
    assert all(pn.distance_bucket(n, rows, most) == rows - 1 for n in (len(got), most, 10 * most))


def test_distance_buckets_at_whole_ratios():
    """8 rows, 4 of one distance each, then half an octave per row: edges at exact powers of two belong to the row above."""
    from ullm_b200.parts.position import distance_buckets

    b = distance_buckets(16, 128)  # rows 8 .. 15 from distances 8 * 2^(i / 2)
    assert [b[n] for n in (8, 15, 16, 31, 32, 63, 64)] == [8, 9, 10, 11, 12, 13, 14]
    with pytest.raises(ValueError):
        distance_buckets(1, 5)
    with pytest.raises(ValueError):
        distance_buckets(8, 4)


@pytest.mark.parametrize("change,needle", [
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["norm"].update(eps=0), "eps"),
    (lambda c: c.update(logit_scale="1"), "logit_scale"),
    (lambda c: c["embedding"]["bigram"].update(buckets=0), "buckets"),
    (lambda c: c["embedding"]["bigram"].pop("mul_prev"), "mul_prev"),
    (lambda c: c["embedding"]["bigram"].update(mul_cur=1.5), "mul_cur"),
    (lambda c: c["layers"][0].update(type="attention"), "type"),
    (lambda c: c["layers"][0].pop("mixer"), "mixer"),
    (lambda c: c["layers"][0]["mixer"].pop("left"), "heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(bias_max=5), "bias_max"),
    (lambda c: c["layers"][0]["mixer"]["left"]["q_temp"].update(every=0), "every"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("state"), "state"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(groups=3), "groups"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][1]["mixer"].pop("dim"), "dim"),
    (lambda c: c["layers"][2]["mixer"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][2]["mixer"].update(decay=[0.5, 1.5]), "decay"),
    (lambda c: c["layers"][2]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][1]["mlp"].update(kind="gated"), "kind"),
    (lambda c: c["layers"][1]["mlp"].pop("ff"), "ff"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "top"),
])
def test_config_errors_name_the_key(change, needle):
    from ullm_b200.config.ninelix import NinelixConfig, NinelixConfigError

    cfg = copy.deepcopy(CFG_A)
    change(cfg)
    with pytest.raises(NinelixConfigError, match=needle):
        NinelixConfig.from_dict(cfg, _shapes("A"))


def test_sizes_that_only_tensors_give(tmp_path):
    from ullm_b200.config import load_model_spec
    from ullm_b200.config.ninelix import NinelixConfig, NinelixConfigError

    cfg, w, _ = weights_for("C", "bfloat16")
    typed, spec = load_model_spec(write_model(str(tmp_path / "m"), cfg, w))
    assert [L.decay_rank for L in typed.layers] == [None, None, 5, None, 70]
    assert [L.bias_rows for L in typed.layers] == [None, 9, None, 4, None]
    assert spec.layers[2].mixer.args["decay_rank"] == 5
    shapes = _shapes("C")
    shapes.pop("l2.mix.w1")
    with pytest.raises(NinelixConfigError, match="l2.mix.w1"):
        NinelixConfig.from_dict(cfg, shapes)
    assert NinelixConfig.from_dict(config(32, 40, [wkv(2, 8)])).layers[0].decay_rank > 0  # (no files: a default)


def test_random_model_folder_round_trip(tmp_path):
    from ullm_b200.config import load_model_spec
    from ullm_b200.engine.cli import main
    from ullm_b200.weights.safetensors_io import open_model_files

    cfg = config(40, 50, [wkv(2, 8, dense(24)), lightning(8, 12, [0.5, 0.9]), parallel(left(2, 1, 8, 8, 0.3, 2, 64), right(2, 8, 4, 1, 3, 1))])
    path = tmp_path / "cfg.json"
    path.write_text(json.dumps(cfg))
    out = str(tmp_path / "model")
    assert main(["random-model", "--out", out, "--config", str(path), "--seed", "3", "--dtype", "bfloat16"]) == 0
    files = open_model_files(out)
    shapes = {n: tuple(f.shape(n)) for f in files for n in f.names()}
    for f in files:
        f.close()
    rank, rows = shapes["l0.mix.w1"][0], shapes["l2.mix.left.rel"][0]
    assert shapes == {n: tuple(s) for n, (s, _) in pn.tensor_shapes(cfg, decay_rank=rank, bias_rows=rows).items()}
    typed, spec = load_model_spec(out)
    assert spec.architecture == "Ninelix" and typed.to_dict()["layers"] == cfg["layers"]


def test_state_rows_and_pages_that_the_layers_ask_for():
    from ullm_b200.cache.manager import CacheManager, plan_groups_with_aux

    needs = _model("A").cache_needs()
    assert [n[0] is not None for n in needs] == [True, False, False, False, False, True, False]
    assert all(n[1] is not None for n in needs)  # every layer keeps state, and so does the embedding (the last entry)
    up = lambda n: -(-n // 4) * 4
    assert needs[0][1].shape == (up(2 * (4 * 24 + 2 * 24 + 2 * 40)) + up(4 * 12 * 20) + up(3 * (48 + 80)),)
    assert needs[1][1].shape == (3 * 24 * 24 + 72,) and needs[2][1].shape == (2 * 20 * 28,)
    assert needs[6][1].shape == (1,) and needs[6][1].dtype == torch.int32
    groups, where, _ = plan_groups_with_aux(needs)
    assert len(groups) == 2 and where[6] is None
    c = CacheManager(needs, 8, 12, 2, 6, device="cpu", enable_prefix_cache=True)
    assert c.tree is None  # state: shared pages would not hold all of a prefix
    rc = c.admit("a")
    for s in c.states.values():
        s[rc.slot] = 3
    c.reserve(rc, 9)
    c.commit(rc, 9)
    c.release(rc)
    again = c.admit("b")
    assert again.slot == rc.slot and all(not s[again.slot].any() for s in c.states.values())
    caches = c.layer_caches([None, None])
    assert len(caches) == 7 and caches[6].state.shape == (2, 1)
    # a convolution of one tap keeps no rows: the state-space mixer's part is then the whole row
    d = _model("D").cache_needs()
    assert d[0][1].shape == (16,) and d[3][1].shape == (up(2 * 24) + up(2 * (2 + 96)),)


# ---------------------------------------------------------------------------------------------------------
# the plain implementation's own reading
# ---------------------------------------------------------------------------------------------------------
def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


def test_plain_pair_embedding():
    cfg = config(8, 20, [wkv(1, 4)], buckets=7, mul_prev=11, mul_cur=4)
    w = pn.random_weights(cfg, seed=1)
    x = pn.embed([3, 19, 3], w, cfg)
    assert torch.equal(x[0], w["embed"][3] + w["bigram"][7])
    assert torch.equal(x[1], w["embed"][19] + w["bigram"][(33 + 76) % 7])
    assert torch.equal(x[2], w["embed"][3] + w["bigram"][(11 * 19 + 12) % 7])


def test_plain_wkv_bonus_is_for_the_current_token_alone():
    n, H, d = 4, 2, 3
    r, k, v = (rnd(n, H, d, seed=s) for s in range(3))
    w = torch.rand(n, H, d, generator=torch.Generator().manual_seed(5), dtype=torch.float64)
    u = rnd(H, d, seed=7)
    o = pn.wkv_core(r, k, v, w, u)
    for t in range(n):
        for h in range(H):
            want = (r[t, h] * u[h] * k[t, h]).sum() * v[t, h]
            for s in range(t):
                decay = torch.ones(d, dtype=torch.float64)
                for q in range(s + 1, t):
                    decay = decay * w[q, h]
                want = want + (r[t, h] * decay * k[s, h]).sum() * v[s, h]
            assert torch.allclose(o[t, h], want)


def test_plain_fixed_decay_counts_the_current_token_undecayed():
    q, k, v = rnd(3, 1, 2), rnd(3, 1, 2, seed=1), rnd(3, 1, 4, seed=2)
    o = pn.fixed_decay_core(q, k, v, [0.5])
    want = sum(0.5 ** (2 - s) * (q[2, 0] @ k[s, 0]) * v[s, 0] for s in range(3))
    assert torch.allclose(o[2, 0], want)


def test_plain_attention_bias_is_not_scaled_and_the_temperature_steps():
    q, k, v = rnd(2, 3, 4), rnd(1, 3, 4, seed=1), rnd(1, 3, 2, seed=2)
    rel = rnd(4, 2, seed=3)
    a = pn.biased_attention_core(q, k, v, 0.3, rel, 9)
    s = torch.stack([0.3 * (q[1, 2] @ k[0, j]) + rel[pn.distance_bucket(2 - j, 4, 9), 1] for j in range(3)])
    assert torch.allclose(a[2, 1], torch.softmax(s, 0) @ v[0])
    assert pn.query_temperature(6, 0.5, 8) == 1.0 and pn.query_temperature(7, 0.5, 8) == 1.0 + 0.5 * math.log(2)
    assert pn.query_temperature(15, 0.5, 8) == 1.0 + 0.5 * math.log(3)


def test_plain_token_shift_and_convolution_see_zeros_in_front():
    h = rnd(3, 5)
    assert not pn.token_shift(h)[0].any() and torch.equal(pn.token_shift(h)[1:], h[:-1])
    w = rnd(5, 3, seed=4)
    y = pn.causal_conv(h, w)
    assert torch.allclose(y[0], w[:, 2] * h[0]) and torch.allclose(y[2], w[:, 0] * h[0] + w[:, 1] * h[1] + w[:, 2] * h[2])


def test_plain_choice_is_a_softmax_over_the_chosen():
    h = rnd(4, 6)
    w = {"router": rnd(5, 6, seed=2)}
    chosen, weight = pn.route(h, w, "", dict(experts=5, top=2))
    z = h @ w["router"].T
    assert torch.allclose(weight.sum(-1), torch.ones(4, dtype=torch.float64))
    assert torch.equal(chosen, torch.topk(z, 2).indices)
    p = torch.softmax(z, -1).gather(1, chosen)
    assert torch.allclose(weight, p / p.sum(-1, keepdim=True))


def test_plain_prefix_does_not_see_what_follows():
    for cfg, tag in ((CFG_B, "B"), (CFG_C, "C"), (CFG_E, "E")):
        _, w, _ = weights_for(tag, "float32")
        ids = [(7 * i + i * i) % cfg["vocab"] for i in range(24)]
        a = oracle(ids, w, cfg)
        b = oracle(ids[:15], w, cfg)
        assert torch.allclose(a[:15], b, atol=1e-5)
