"""Typed configuration of the Ninelix decoder, read from the keys of its config.json, and its translation into a
ModelSpec.

The design: a token embedding to which a second table adds a row that the token and the one before it choose together
(`embedding.bigram`); a list of layers on a 32-bit residual stream whose norms sit on the sub-layers' outputs only,
x <- x + norm1(mixer(x)) and, if the layer has a feed-forward, x <- x + norm2(ff(x)), RMS norms whose stored weight is around
zero (1 + w); an output head of its own whose logits are multiplied by `logit_scale`.  Three mixers:

* wkv: time mixing with a decay per key channel and a bonus for the current token (parts/wkv.py).
* lightning: linear attention with one fixed decay per head (parts/lightning.py).
* parallel: two mixers read the same rows, each one's output is RMS-normed over the model width with a weight of its own,
  and the result is half the sum.  left: grouped causal attention with biases on q, k and v, a short convolution on each of
  their channels, an RMS norm per head on q and k, no rotation, a query temperature that grows with the position, a learned
  bias per distance bucket and head, and an output gate of one number per head.  right: a state-space recurrence with a
  scalar decay per head (Mamba-2).

Feed-forward `dense`: W_down gelu(W_up h) with the exact gelu; `moe`: gated silu experts of which each token takes the `top`
with the largest router logits, weighted by a softmax over the chosen ones.

config.json keys: architecture, vocab, width, logit_scale, norm.eps, embedding.bigram{buckets, mul_prev, mul_cur}, layers[]
with type, mixer (wkv: heads, dim; lightning: heads, dim, vdim, decay[]; parallel: left{heads, kv_heads, dim, vdim, conv,
scale, q_temp{coef, every}, bias_max}, right{heads, vdim, state, groups, conv, norm_groups}),
mlp{kind: dense, ff} | {kind: moe, expert{ff}, router{experts, top}} | null.  Two sizes are given by tensors alone: the rank
of a wkv layer's decay ('.w1') and the rows of an attention's distance table ('.rel').
Tensor names: embed, bigram, l<i>.norm1, l<i>.norm2, l<i>.mix.*, l<i>.mlp.*, final.norm, head.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any

from .specs import FeedForwardSpec, LayerSpec, MixerSpec, ModelSpec, NormSpec, PairEmbeddingSpec, ScheduleEntry

ARCHITECTURE = "Ninelix"
MIXER_TYPES = ("wkv", "lightning", "parallel")
# sizes that only tensors give, for folders without weight files (random weights)
DEFAULT_DECAY_RANK = 64
DEFAULT_BIAS_ROWS = 32


class NinelixConfigError(ValueError):
    pass


def _need(d, key: str, where: str, kind=(int, float)):
    if not isinstance(d, dict) or key not in d:
        raise NinelixConfigError(f"config.json: {where} lacks {key!r}")
    v = d[key]
    if isinstance(v, bool) or not isinstance(v, kind):
        raise NinelixConfigError(f"config.json: {where}.{key} = {v!r} is not a number")
    return v


def _positive_int(d, key: str, where: str) -> int:
    v = _need(d, key, where, (int,))
    if v <= 0:
        raise NinelixConfigError(f"config.json: {where}.{key} must be positive, got {v}")
    return v


def _positive(d, key: str, where: str) -> float:
    v = float(_need(d, key, where))
    if not v > 0:
        raise NinelixConfigError(f"config.json: {where}.{key} must be positive, got {v}")
    return v


def _check_wkv(m, where: str) -> None:
    for k in ("heads", "dim"):
        _positive_int(m, k, where)


def _check_lightning(m, where: str) -> None:
    for k in ("heads", "dim", "vdim"):
        _positive_int(m, k, where)
    d = m.get("decay")
    if (not isinstance(d, list) or len(d) != m["heads"]
            or not all(isinstance(v, (int, float)) and not isinstance(v, bool) and 0.0 < v <= 1.0 for v in d)):
        raise NinelixConfigError(f"config.json: {where}.decay must list one number above 0 and at most 1 per head")


def _check_left(left, where: str) -> None:
    for k in ("heads", "kv_heads", "dim", "vdim", "bias_max", "conv"):
        _positive_int(left, k, where)
    if left["heads"] % left["kv_heads"]:
        raise NinelixConfigError(f"config.json: {where}.heads is no multiple of kv_heads")
    _need(left, "scale", where)
    t = left.get("q_temp")
    if t is not None:
        _need(t, "coef", where + ".q_temp")
        _positive_int(t, "every", where + ".q_temp")


def _check_right(right, where: str) -> None:
    for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups"):
        _positive_int(right, k, where)
    if right["heads"] % right["groups"]:
        raise NinelixConfigError(f"config.json: {where}.heads is no multiple of groups")
    if (right["heads"] * right["vdim"]) % right["norm_groups"]:
        raise NinelixConfigError(f"config.json: {where}: heads x vdim is no multiple of norm_groups")


def _check_mlp(mlp, where: str) -> None:
    kind = mlp.get("kind") if isinstance(mlp, dict) else None
    if kind == "dense":
        _positive_int(mlp, "ff", where)
        return
    if kind != "moe":
        raise NinelixConfigError(f"config.json: {where}.kind must be 'dense' or 'moe'")
    _positive_int(mlp.get("expert"), "ff", where + ".expert")
    r, rw = mlp.get("router"), where + ".router"
    if _positive_int(r, "top", rw) > _positive_int(r, "experts", rw):
        raise NinelixConfigError(f"config.json: {rw}.top is more than there are experts")


def _rows_of(shapes, name: str, default: int) -> int:
    """The first dimension of a tensor, where the model folder has weight files."""
    if shapes is None:
        return default
    if name not in shapes or len(shapes[name]) != 2:
        raise NinelixConfigError(f"the model folder has no matrix {name!r}, whose rows are a size of the model")
    return int(shapes[name][0])


@dataclass(frozen=True)
class NinelixLayer:
    type: str
    mixer: dict[str, Any]
    mlp: dict[str, Any] | None
    decay_rank: int | None = None  # wkv
    bias_rows: int | None = None  # parallel


@dataclass(frozen=True)
class NinelixConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_scale: float
    bigram: tuple[int, int, int] | None  # buckets, mul_prev, mul_cur
    layers: tuple[NinelixLayer, ...]
    dtype: str = "bfloat16"
    max_positions: int = 1 << 30  # nothing is tabulated by position: the context is the engine's choice
    raw: dict[str, Any] = field(default_factory=dict, hash=False, compare=False)

    @staticmethod
    def from_dict(d: dict[str, Any], shapes: dict[str, tuple] | None = None) -> "NinelixConfig":
        vocab, width = _positive_int(d, "vocab", "the config"), _positive_int(d, "width", "the config")
        eps = _positive(d.get("norm"), "eps", "norm")
        logit_scale = float(_need(d, "logit_scale", "the config")) if "logit_scale" in d else 1.0
        b = (d.get("embedding") or {}).get("bigram")
        bigram = None
        if b is not None:
            where = "embedding.bigram"
            bigram = (_positive_int(b, "buckets", where), int(_need(b, "mul_prev", where, (int,))),
                      int(_need(b, "mul_cur", where, (int,))))
        raw_layers = d.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise NinelixConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(raw_layers):
            where = f"layers[{i}]"
            if not isinstance(L, dict) or L.get("type") not in MIXER_TYPES:
                raise NinelixConfigError(f"config.json: {where}.type must be one of {MIXER_TYPES}")
            mix, wm = L.get("mixer"), where + ".mixer"
            if not isinstance(mix, dict):
                raise NinelixConfigError(f"config.json: {where} lacks 'mixer'")
            rank = rows = None
            if L["type"] == "wkv":
                _check_wkv(mix, wm)
                rank = _rows_of(shapes, f"l{i}.mix.w1", DEFAULT_DECAY_RANK)
            elif L["type"] == "lightning":
                _check_lightning(mix, wm)
            else:
                _check_left(mix.get("left"), wm + ".left")
                _check_right(mix.get("right"), wm + ".right")
                rows = _rows_of(shapes, f"l{i}.mix.left.rel", DEFAULT_BIAS_ROWS)
                if rows < 2 or mix["left"]["bias_max"] <= rows // 2:
                    raise NinelixConfigError(f"config.json: {wm}.left.bias_max must lie above half the rows of the distance "
                                             f"table ({rows}, at least 2)")
            mlp = L.get("mlp")
            if mlp is not None:
                _check_mlp(mlp, where + ".mlp")
            layers.append(NinelixLayer(L["type"], dict(mix), dict(mlp) if mlp is not None else None, rank, rows))
        dt = str(d.get("dtype", d.get("torch_dtype", "bfloat16"))).replace("torch.", "")
        if dt not in ("bfloat16", "float32", "float16"):
            raise NinelixConfigError(f"Unsupported dtype {dt!r}")
        return NinelixConfig(vocab, width, eps, logit_scale, bigram, tuple(layers), dt, raw=dict(d))

    def to_dict(self) -> dict[str, Any]:
        return dict(self.raw)


def _mixer(L: NinelixLayer, W: int, eps: float) -> MixerSpec:
    m = L.mixer
    if L.type == "wkv":
        return MixerSpec("wkv", dict(
            hidden_size=W, num_heads=m["heads"], head_dim=m["dim"], decay_rank=L.decay_rank, eps=eps,
            names=dict(mu="mu.{}", r="r", k="k", v="v", g="g", w1="w1", w2="w2", w0="w0", u="u", norm="norm", o="o")))
    if L.type == "lightning":
        return MixerSpec("fixed_decay_attention", dict(
            hidden_size=W, num_heads=m["heads"], head_dim=m["dim"], value_dim=m["vdim"], decay=list(m["decay"]), eps=eps,
            names=dict(q="q", k="k", v="v", gate="g", o="o", norm="norm")))
    a, s = m["left"], m["right"]
    t = a.get("q_temp")
    left = MixerSpec("paged_attention", dict(
        hidden_size=W, num_heads=a["heads"], num_kv_heads=a["kv_heads"], head_dim=a["dim"], value_dim=a["vdim"],
        qkv_bias=True, conv_taps=a["conv"], qk_norm=NormSpec("rmsnorm", a["dim"], eps, dict(param="")),
        q_temperature=(float(t["coef"]), t["every"]) if t is not None else None,
        distance_bias=(L.bias_rows, a["bias_max"]), head_gate=True, scale=float(a["scale"]),
        names=dict(q="q", k="k", v="v", o="o", q_bias="q.b", k_bias="k.b", v_bias="v.b", q_norm="q.norm", k_norm="k.norm",
                   q_conv="q.conv", k_conv="k.conv", v_conv="v.conv", rel="rel", gate="g")))
    right = MixerSpec("mamba2", dict(
        hidden_size=W, num_heads=s["heads"], value_dim=s["vdim"], state=s["state"], groups=s["groups"],
        conv_taps=s["conv"], norm_groups=s["norm_groups"], eps=eps,
        names=dict(in_proj="in", conv="conv", conv_bias="conv.b", dt_bias="dt_bias", a_log="A_log", d="D", norm="norm",
                   o="o")))
    return MixerSpec("parallel_normed_mixers", dict(
        hidden_size=W, left=left, right=right, eps=eps, mult=0.5,
        names=dict(left="left.", right="right.", left_norm="left.out", right_norm="right.out")))


def _feed_forward(f: dict, W: int) -> FeedForwardSpec:
    if f["kind"] == "dense":
        return FeedForwardSpec("dense_mlp", dict(hidden_size=W, intermediate_size=f["ff"], activation="gelu",
                                                 names=dict(up="up", down="down")))
    r = f["router"]
    # (a softmax over all logits, renormalized over the chosen ones, is the softmax over the chosen ones)
    return FeedForwardSpec("routed_experts", dict(
        hidden_size=W, intermediate_size=f["expert"]["ff"], num_experts=r["experts"], top=r["top"], activation="silu",
        scores="softmax", renormalize=True, weight_on="output",
        names=dict(router="router", gate="e{}.gate", up="e{}.up", down="e{}.down")))


def ninelix_model_spec(cfg: NinelixConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps

    def norm():
        return NormSpec("rmsnorm", W, eps, dict(param="", around_zero=True))

    layers = []
    for L in cfg.layers:
        ff = _feed_forward(L.mlp, W) if L.mlp is not None else None
        layers.append(LayerSpec(
            block="outnorm_residual", mixer=_mixer(L, W, eps), feed_forward=ff, mixer_norm=norm(),
            feed_forward_norm=norm() if ff is not None else None,
            names=dict(mixer="mix.", feed_forward="mlp.", mixer_norm="norm1", feed_forward_norm="norm2")))
    pairs = PairEmbeddingSpec("bigram", *cfg.bigram) if cfg.bigram is not None else None
    return ModelSpec(
        architecture=ARCHITECTURE, hidden_size=W, vocab_size=cfg.vocab, layers=layers,
        schedule=[ScheduleEntry(i) for i in range(len(layers))], final_norm=norm(), tie_embeddings=False,
        max_positions=cfg.max_positions, dtype=cfg.dtype, embedding_name="embed", layer_name="l{}.",
        final_norm_name="final.norm", head_name="head", embedding_param="", head_param="", stream_dtype="float32",
        embedding_pairs=pairs, logit_scale=cfg.logit_scale)
