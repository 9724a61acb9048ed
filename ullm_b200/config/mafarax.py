"""Typed configuration of the Mafarax decoder, read from the keys of its config.json, and its translation into a
ModelSpec.

The design: a token embedding and an output head of its own; a list of pre-norm layers on a 32-bit residual stream,
x <- x + mixer(norm1(x)) and, if the layer has a feed-forward, x <- x + ff(norm2(x)), where the norm is a tanh without
statistics, tanh(alpha x) * w + b; logits times `logit_scale`.  The mixer of every layer is `parallel`: two mixers read the
same rows, each one's output is RMS-normed over the model width with a weight of its own, and the result is half the sum.

* left: grouped-query attention with biases on all four projections; the first `rot.dims` dimensions of q and k turn in
  halves (i, i + dims / 2) with frequencies divided by `rot.scaling.factor`; position i sees the j <= i of its own stretch of
  `mask.size` positions, stretches being counted from position 0.
* right: a state-space recurrence with a scalar decay per head (Mamba-2): a short convolution with silu, per-request state,
  a silu gate in front of an RMS norm over `norm_groups` equal parts.

Feed-forward `moe`: `experts` routed experts W_down relu(W_up h)^2, of which each token takes `top`; sigmoid scores; the
experts form `groups.count` groups, of which the `groups.keep` best (by the sum of the two largest scores) can be chosen
from; weights times `scale`, not renormalized; a shared expert of the same form runs for every token.

config.json keys: architecture, vocab, width, logit_scale, norm.eps, layers[] with type, mixer{left{heads, kv_heads, dim,
vdim, scale, mask{size}, rot{base, dims, scaling{factor}}}, right{heads, vdim, state, groups, conv, norm_groups}},
mlp{kind, expert{ff}, router{experts, top, scale, groups{count, keep}}, shared{ff} | null} | null.
Tensor names: embed, l<i>.norm1, l<i>.norm2 (each with .alpha and .b), l<i>.mix.left.*, l<i>.mix.right.*, l<i>.mlp.*,
final.norm, head.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any

from .specs import FeedForwardSpec, LayerSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec, ScheduleEntry

ARCHITECTURE = "Mafarax"
MIXER_TYPES = ("parallel",)


class MafaraxConfigError(ValueError):
    pass


def _need(d, key: str, where: str, kind=(int, float)):
    if not isinstance(d, dict) or key not in d:
        raise MafaraxConfigError(f"config.json: {where} lacks {key!r}")
    v = d[key]
    if isinstance(v, bool) or not isinstance(v, kind):
        raise MafaraxConfigError(f"config.json: {where}.{key} = {v!r} is not a number")
    return v


def _positive_int(d, key: str, where: str) -> int:
    v = _need(d, key, where, (int,))
    if v <= 0:
        raise MafaraxConfigError(f"config.json: {where}.{key} must be positive, got {v}")
    return v


def _positive(d, key: str, where: str) -> float:
    v = float(_need(d, key, where))
    if not v > 0:
        raise MafaraxConfigError(f"config.json: {where}.{key} must be positive, got {v}")
    return v


def _stretch(left: dict, where: str) -> int | None:
    """The size of the stretches of positions that see one another; None without a mask."""
    mask = left.get("mask")
    return None if mask is None else _positive_int(mask, "size", where + ".mask")


def _rotation(left: dict, where: str) -> PositionSpec | None:
    rot = left.get("rot")
    if rot is None:
        return None
    dims = _positive_int(rot, "dims", where + ".rot")
    if dims % 2 or dims > left["dim"]:
        raise MafaraxConfigError(f"config.json: {where}.rot.dims must be even and at most dim")
    args = {}
    if rot.get("scaling") is not None:
        args["scaling"] = dict(factor=_positive(rot["scaling"], "factor", where + ".rot.scaling"))
    return PositionSpec("rope_computed", rotary_dim=dims, theta=_positive(rot, "base", where + ".rot"), args=args)


def _check_left(left, where: str) -> None:
    for k in ("heads", "kv_heads", "dim", "vdim"):
        _positive_int(left, k, where)
    if left["heads"] % left["kv_heads"]:
        raise MafaraxConfigError(f"config.json: {where}.heads is no multiple of kv_heads")
    _need(left, "scale", where)
    _stretch(left, where)
    _rotation(left, where)


def _check_right(right, where: str) -> None:
    for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups"):
        _positive_int(right, k, where)
    if right["heads"] % right["groups"]:
        raise MafaraxConfigError(f"config.json: {where}.heads is no multiple of groups")
    if (right["heads"] * right["vdim"]) % right["norm_groups"]:
        raise MafaraxConfigError(f"config.json: {where}: heads x vdim is no multiple of norm_groups")


def _router_groups(router: dict, where: str) -> tuple[int, int] | None:
    g = router.get("groups")
    if g is None:
        return None
    count, keep = _positive_int(g, "count", where + ".groups"), _positive_int(g, "keep", where + ".groups")
    if router["experts"] % count or keep > count or router["top"] > keep * (router["experts"] // count):
        raise MafaraxConfigError(f"config.json: {where}.groups: {count} equal groups of {router['experts']} experts, of "
                                 f"which {keep} must hold at least top = {router['top']}")
    return count, keep


def _check_mlp(mlp, where: str) -> None:
    if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
        raise MafaraxConfigError(f"config.json: {where}.kind must be 'moe'")
    _positive_int(mlp.get("expert"), "ff", where + ".expert")
    r, rw = mlp.get("router"), where + ".router"
    E, top = _positive_int(r, "experts", rw), _positive_int(r, "top", rw)
    if top > E:
        raise MafaraxConfigError(f"config.json: {rw}.top is more than there are experts")
    if "scale" in r:
        _need(r, "scale", rw)
    _router_groups(r, rw)
    if mlp.get("shared") is not None:
        _positive_int(mlp["shared"], "ff", where + ".shared")


@dataclass(frozen=True)
class MafaraxLayer:
    type: str
    mixer: dict[str, Any]
    mlp: dict[str, Any] | None


@dataclass(frozen=True)
class MafaraxConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_scale: float
    layers: tuple[MafaraxLayer, ...]
    dtype: str = "bfloat16"
    max_positions: int = 1 << 30  # positions are computed, not tabulated: the context is the engine's choice
    raw: dict[str, Any] = field(default_factory=dict, hash=False, compare=False)

    @staticmethod
    def from_dict(d: dict[str, Any]) -> "MafaraxConfig":
        vocab, width = _positive_int(d, "vocab", "the config"), _positive_int(d, "width", "the config")
        eps = _positive(d.get("norm"), "eps", "norm")
        logit_scale = float(_need(d, "logit_scale", "the config")) if "logit_scale" in d else 1.0
        raw_layers = d.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise MafaraxConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(raw_layers):
            where = f"layers[{i}]"
            if not isinstance(L, dict) or L.get("type") not in MIXER_TYPES:
                raise MafaraxConfigError(f"config.json: {where}.type must be one of {MIXER_TYPES}")
            mix = L.get("mixer")
            if not isinstance(mix, dict):
                raise MafaraxConfigError(f"config.json: {where} lacks 'mixer'")
            _check_left(mix.get("left"), where + ".mixer.left")
            _check_right(mix.get("right"), where + ".mixer.right")
            mlp = L.get("mlp")
            if mlp is not None:
                _check_mlp(mlp, where + ".mlp")
            layers.append(MafaraxLayer(L["type"], dict(mix), dict(mlp) if mlp is not None else None))
        dt = str(d.get("dtype", d.get("torch_dtype", "bfloat16"))).replace("torch.", "")
        if dt not in ("bfloat16", "float32", "float16"):
            raise MafaraxConfigError(f"Unsupported dtype {dt!r}")
        return MafaraxConfig(vocab, width, eps, logit_scale, tuple(layers), dt, raw=dict(d))

    def to_dict(self) -> dict[str, Any]:
        return dict(self.raw)


def _mixer(mix: dict, W: int, eps: float) -> MixerSpec:
    a, s = mix["left"], mix["right"]
    left = MixerSpec("paged_attention", dict(
        hidden_size=W, num_heads=a["heads"], num_kv_heads=a["kv_heads"], head_dim=a["dim"], value_dim=a["vdim"],
        qkv_bias=True, o_bias=True, position=_rotation(a, "mixer.left"), chunk=_stretch(a, "mixer.left"),
        scale=float(a["scale"]), general=True,
        names=dict(q="q", k="k", v="v", o="o", q_bias="q.b", k_bias="k.b", v_bias="v.b", o_bias="o.b")))
    right = MixerSpec("mamba2", dict(
        hidden_size=W, num_heads=s["heads"], value_dim=s["vdim"], state=s["state"], groups=s["groups"],
        conv_taps=s["conv"], norm_groups=s["norm_groups"], eps=eps,
        names=dict(in_proj="in", conv="conv", conv_bias="conv.b", dt_bias="dt_bias", a_log="A_log", d="D", norm="norm",
                   o="o")))
    return MixerSpec("parallel_normed_mixers", dict(
        hidden_size=W, left=left, right=right, eps=eps, mult=0.5,
        names=dict(left="left.", right="right.", left_norm="left.out", right_norm="right.out")))


def _feed_forward(f: dict, W: int) -> FeedForwardSpec:
    r = f["router"]
    shared = None
    if f.get("shared") is not None:
        shared = FeedForwardSpec("dense_mlp", dict(hidden_size=W, intermediate_size=f["shared"]["ff"], activation="relu2",
                                                   names=dict(up="up", down="down")))
    return FeedForwardSpec("routed_experts", dict(
        hidden_size=W, intermediate_size=f["expert"]["ff"], num_experts=r["experts"], top=r["top"], activation="relu2",
        gated=False, scores="sigmoid", renormalize=False, weight_on="output", groups=_router_groups(r, "mlp.router"),
        weight_scale=float(r.get("scale", 1.0)), shared=shared,
        names=dict(router="router", up="e{}.up", down="e{}.down", shared="shared.")))


def mafarax_model_spec(cfg: MafaraxConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps

    def norm():
        return NormSpec("dynamic_tanh", W, eps, dict(param="", bias_param=".b", alpha_param=".alpha"))

    layers = []
    for L in cfg.layers:
        ff = _feed_forward(L.mlp, W) if L.mlp is not None else None
        layers.append(LayerSpec(
            block="prenorm_scaled", mixer=_mixer(L.mixer, W, eps), feed_forward=ff, mixer_norm=norm(),
            feed_forward_norm=norm() if ff is not None else None,
            names=dict(mixer="mix.", feed_forward="mlp.", mixer_norm="norm1", feed_forward_norm="norm2")))
    return ModelSpec(
        architecture=ARCHITECTURE, hidden_size=W, vocab_size=cfg.vocab, layers=layers,
        schedule=[ScheduleEntry(i) for i in range(len(layers))], final_norm=norm(), tie_embeddings=False,
        max_positions=cfg.max_positions, dtype=cfg.dtype, embedding_name="embed", layer_name="l{}.",
        final_norm_name="final.norm", head_name="head", embedding_param="", head_param="", stream_dtype="float32",
        logit_scale=cfg.logit_scale)
