"""The Ninelix decoder restated plainly: one slow function per mechanism, whole sequences at once, any float dtype (the
tests run it in 64-bit on the weights as given).  It shares no code with the engine.

Notation: n tokens, positions 0 .. n-1; x [n, width]; a linear map is `x @ W.T` with W [out, in].
"""

from __future__ import annotations

import math

import torch


def silu(z):
    return z * torch.sigmoid(z)


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


# ---------------------------------------------------------------------------------------------------------
# norms, embedding
# ---------------------------------------------------------------------------------------------------------
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def rms_norm_one_plus(x, w, eps):
    return unit_rms(x, eps) * (1.0 + w)


def bigram_row(prev, cur, b):
    """Row of the pair (prev, cur); the last row for a first token (prev None)."""
    return b["buckets"] if prev is None else (prev * b["mul_prev"] + cur * b["mul_cur"]) % b["buckets"]


def embed(ids, w, cfg):
    b = cfg["embedding"]["bigram"]
    rows = [bigram_row(ids[t - 1] if t else None, ids[t], b) for t in range(len(ids))]
    return w["embed"][torch.tensor(list(ids))] + w["bigram"][torch.tensor(rows)]


# ---------------------------------------------------------------------------------------------------------
# mixer: time mixing with a decay per key channel and a bonus for the current token
# ---------------------------------------------------------------------------------------------------------
def token_shift(h):
    """h of the token before, zeros in front of the first."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def wkv_core(r, k, v, decay, u):
    """r, k, v, decay [n, H, d], u [H, d] -> [n, H, d]."""
    n, H, d = r.shape
    out = torch.zeros_like(v)
    for h in range(H):
        S = torch.zeros(d, d, dtype=r.dtype)
        for t in range(n):
            kv = torch.outer(k[t, h], v[t, h])
            out[t, h] = (S + u[h][:, None] * kv).T @ r[t, h]
            S = decay[t, h][:, None] * S + kv
    return out


def wkv_mixer(h, m, w, pre, eps):
    n, H, d = h.shape[0], m["heads"], m["dim"]
    before = token_shift(h)
    mix = {s: h + (before - h) * w[f"{pre}mu.{s}"] for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[pre + s].T).reshape(n, H, d) for s in "rkv")
    gate = silu(mix["g"] @ w[pre + "g"].T)
    z = torch.tanh(mix["w"] @ w[pre + "w1"].T) @ w[pre + "w2"].T + w[pre + "w0"]
    decay = torch.exp(-torch.exp(z)).reshape(n, H, d)
    o = unit_rms(wkv_core(r, k, v, decay, w[pre + "u"]), eps).reshape(n, H * d)
    return (o * w[pre + "norm"] * gate) @ w[pre + "o"].T


# ---------------------------------------------------------------------------------------------------------
# mixer: linear attention with one fixed decay per head
# ---------------------------------------------------------------------------------------------------------
def fixed_decay_core(q, k, v, decay):
    """q, k [n, H, d], v [n, H, dv], decay [H] -> [n, H, dv]."""
    n, H, d = q.shape
    out = torch.zeros_like(v)
    for h in range(H):
        S = torch.zeros(d, v.shape[-1], dtype=q.dtype)
        for t in range(n):
            S = decay[h] * S + torch.outer(k[t, h], v[t, h])
            out[t, h] = S.T @ q[t, h]
    return out


def lightning_mixer(h, m, w, pre, eps):
    n, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = (silu(h @ w[pre + s].T).reshape(n, H, d) for s in "qk")
    v = silu(h @ w[pre + "v"].T).reshape(n, H, dv)
    o = fixed_decay_core(q, k, v, m["decay"]).reshape(n, H * dv)
    return (rms_norm(o, w[pre + "norm"], eps) * torch.sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ---------------------------------------------------------------------------------------------------------
# mixer: attention beside a state-space recurrence
# ---------------------------------------------------------------------------------------------------------
def causal_conv(u, taps_w):
    """u [n, channels]; taps_w [channels, taps], the last column meets the current token; zeros before the start."""
    n, taps = u.shape[0], taps_w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < n:
            y[back:] = y[back:] + u[:n - back] * taps_w[:, j]
    return y


def distance_bucket(n, rows, most):
    """One row per distance below rows / 2, then rows that widen with the logarithm of the distance, the last one from
    `most` (or before) on."""
    half = rows // 2
    if n < half:
        return n
    step = math.log(n / half) / math.log(most / half) * (rows - half)
    if abs(step - round(step)) < 1e-9:  # (a power ratio: the floor must not depend on the logarithms' last bit)
        step = round(step)
    return min(rows - 1, half + math.floor(step))


def query_temperature(p, coef, every):
    return 1.0 + coef * math.log((p + 1) // every + 1)


def biased_attention_core(q, k, v, scale, rel=None, most=None):
    """q [H, n, d], k [G, n, d], v [G, n, dv] -> [n, H, dv].  Query i sees every j <= i; rel [rows, H] adds a number per
    distance bucket and head to the scaled score."""
    H, n, _ = q.shape
    G, dv = k.shape[0], v.shape[-1]
    rep = H // G
    out = torch.zeros(n, H, dv, dtype=q.dtype)
    buckets = None
    if rel is not None:
        buckets = torch.tensor([distance_bucket(i, rel.shape[0], most) for i in range(n)])
    for i in range(n):
        s = torch.einsum("hjd,hd->hj", k[:, :i + 1].repeat_interleave(rep, 0), q[:, i]) * scale
        if rel is not None:
            s = s + rel[buckets[:i + 1].flip(0)].T
        out[i] = torch.einsum("hj,hjd->hd", torch.softmax(s, -1), v[:, :i + 1].repeat_interleave(rep, 0))
    return out


def left_mixer(h, m, w, pre, eps):
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def proj(name, heads, size):
        u = h @ w[pre + name].T + w[pre + name + ".b"]
        return causal_conv(u, w[pre + name + ".conv"]).reshape(n, heads, size).transpose(0, 1)

    q = rms_norm(proj("q", H, d), w[pre + "q.norm"], eps)
    k = rms_norm(proj("k", G, d), w[pre + "k.norm"], eps)
    v = proj("v", G, dv)
    t = m["q_temp"]
    temp = torch.tensor([query_temperature(p, t["coef"], t["every"]) for p in range(n)], dtype=h.dtype)
    a = biased_attention_core(q * temp[None, :, None], k, v, m["scale"], w[pre + "rel"], m["bias_max"])
    gate = torch.sigmoid(h @ w[pre + "g"].T)
    return (a * gate[:, :, None]).reshape(n, H * dv) @ w[pre + "o"].T


def state_space_core(x, B, C, dt, a_log, D):
    """x [n, H, P], B and C [n, G, N], dt [n, H] (after the softplus) -> y [n, H, P]."""
    n, H, P = x.shape
    G, N = B.shape[1], B.shape[2]
    rep = H // G
    y = torch.zeros_like(x)
    for h in range(H):
        S = torch.zeros(N, P, dtype=x.dtype)
        for t in range(n):
            S = torch.exp(-torch.exp(a_log[h]) * dt[t, h]) * S + dt[t, h] * torch.outer(B[t, h // rep], x[t, h])
            y[t, h] = S.T @ C[t, h // rep] + D[h] * x[t, h]
    return y


def right_mixer(h, m, w, pre, eps):
    n = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    u = h @ w[pre + "in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w[pre + "conv"]) + w[pre + "conv.b"])
    x = xbc[:, :inner].reshape(n, H, P)
    B = xbc[:, inner:inner + G * N].reshape(n, G, N)
    C = xbc[:, inner + G * N:].reshape(n, G, N)
    dt = torch.nn.functional.softplus(dt + w[pre + "dt_bias"], threshold=200.0)
    y = state_space_core(x, B, C, dt, w[pre + "A_log"], w[pre + "D"]).reshape(n, inner) * silu(z)
    y = unit_rms(y.reshape(n, m["norm_groups"], -1), eps).reshape(n, inner) * w[pre + "norm"]
    return y @ w[pre + "o"].T


def parallel_mixer(h, m, w, pre, eps):
    left = left_mixer(h, m["left"], w, pre + "left.", eps)
    right = right_mixer(h, m["right"], w, pre + "right.", eps)
    return 0.5 * (rms_norm(left, w[pre + "left.out"], eps) + rms_norm(right, w[pre + "right.out"], eps))


def mixer(h, L, w, pre, eps):
    return dict(wkv=wkv_mixer, lightning=lightning_mixer, parallel=parallel_mixer)[L["type"]](h, L["mixer"], w, pre, eps)


# ---------------------------------------------------------------------------------------------------------
# feed-forward
# ---------------------------------------------------------------------------------------------------------
def dense_ff(h, w, pre):
    return gelu_erf(h @ w[pre + "up"].T) @ w[pre + "down"].T


def expert(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def route(h, w, pre, r):
    """(chosen [n, top], their weights [n, top]): the largest logits (ties go to the lower index), softmax over them."""
    z = h @ w[pre + "router"].T
    chosen = torch.stack([torch.tensor(sorted(range(r["experts"]), key=lambda e: (-float(row[e]), e))[:r["top"]]) for row in z])
    return chosen, torch.softmax(torch.gather(z, 1, chosen), -1)


def routed_ff(h, f, w, pre):
    chosen, weight = route(h, w, pre, f["router"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(chosen.shape[1]):
            y[t] += weight[t, j] * expert(h[t:t + 1], w, f"{pre}e{int(chosen[t, j])}.")[0]
    return y


def feed_forward(h, f, w, pre):
    return dense_ff(h, w, pre) if f["kind"] == "dense" else routed_ff(h, f, w, pre)


# ---------------------------------------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------------------------------------
def layer(x, i, cfg, w, rounded=lambda v: v):
    L, eps, pre = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}."
    x = x + rms_norm_one_plus(rounded(mixer(rounded(x), L, w, pre + "mix.", eps)), w[pre + "norm1"], eps)
    if L.get("mlp") is not None:
        x = x + rms_norm_one_plus(rounded(feed_forward(rounded(x), L["mlp"], w, pre + "mlp.")), w[pre + "norm2"], eps)
    return x


def forward(cfg, w, ids, return_layers: bool = False, rounded=lambda v: v):
    """Logits [n, vocab] of one sequence (and the stream after every layer, if asked).  `rounded`: what happens to the
    sub-layers' inputs and outputs (a rounding to 16 bits shows how far such roundings alone carry)."""
    x = embed(list(ids), w, cfg)
    seen = []
    for i in range(len(cfg["layers"])):
        x = layer(x, i, cfg, w, rounded)
        seen.append(x)
    logits = (rounded(rms_norm_one_plus(x, w["final.norm"], cfg["norm"]["eps"])) @ w["head"].T) * cfg["logit_scale"]
    return (logits, torch.stack(seen)) if return_layers else logits


# ---------------------------------------------------------------------------------------------------------
# shapes and random weights
# ---------------------------------------------------------------------------------------------------------
def tensor_shapes(cfg, decay_rank=12, bias_rows=10):
    """{name: (shape, kind)}.  `decay_rank` and `bias_rows` are sizes that no config key gives (a list: one per layer).
    Kinds: "matrix", "router", "embed", "norm" (near 1), "small" (near 0), "mu" (between 0 and 1), "conv", "rel", "a_log",
    "dt_bias", "w0" (logarithms of decay rates)."""
    W, out = cfg["width"], {}

    def pick(v, i):
        return v[i] if isinstance(v, (list, tuple)) else v

    out["embed"] = ((cfg["vocab"], W), "embed")
    out["bigram"] = ((cfg["embedding"]["bigram"]["buckets"] + 1, W), "embed")
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", L["mixer"]
        out[f"l{i}.norm1"] = ((W,), "small")
        if L["type"] == "wkv":
            H, d, R = m["heads"], m["dim"], pick(decay_rank, i)
            for s in "rkvgw":
                out[f"{p}mu.{s}"] = ((W,), "mu")
            for s in "rkvg":
                out[p + s] = ((H * d, W), "matrix")
            out[p + "w1"] = ((R, W), "matrix")
            out[p + "w2"] = ((H * d, R), "matrix")
            out[p + "w0"] = ((H * d,), "w0")
            out[p + "u"] = ((H, d), "small")
            out[p + "norm"] = ((H * d,), "norm")
            out[p + "o"] = ((W, H * d), "matrix")
        elif L["type"] == "lightning":
            H, d, dv = m["heads"], m["dim"], m["vdim"]
            for s, rows in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv)):
                out[p + s] = ((rows, W), "matrix")
            out[p + "norm"] = ((H * dv,), "norm")
            out[p + "o"] = ((W, H * dv), "matrix")
        else:
            a, pl = m["left"], p + "left."
            H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            for s, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
                out[pl + s] = ((rows, W), "matrix")
                out[f"{pl}{s}.b"] = ((rows,), "small")
                out[f"{pl}{s}.conv"] = ((rows, a["conv"]), "conv")
            out[pl + "q.norm"] = ((d,), "norm")
            out[pl + "k.norm"] = ((d,), "norm")
            out[pl + "rel"] = ((pick(bias_rows, i), H), "rel")
            out[pl + "g"] = ((H, W), "matrix")
            out[pl + "o"] = ((W, H * dv), "matrix")
            s, pr = m["right"], p + "right."
            Hs, P, N, Gs = s["heads"], s["vdim"], s["state"], s["groups"]
            inner, ch = Hs * P, Hs * P + 2 * Gs * N
            out[pr + "in"] = ((inner + ch + Hs, W), "matrix")
            out[pr + "conv"] = ((ch, s["conv"]), "conv")
            out[pr + "conv.b"] = ((ch,), "small")
            out[pr + "dt_bias"] = ((Hs,), "dt_bias")
            out[pr + "A_log"] = ((Hs,), "a_log")
            out[pr + "D"] = ((Hs,), "norm")
            out[pr + "norm"] = ((inner,), "norm")
            out[pr + "o"] = ((W, inner), "matrix")
            out[pl + "out"] = ((W,), "norm")
            out[pr + "out"] = ((W,), "norm")
        f = L.get("mlp")
        if f is None:
            continue
        out[f"l{i}.norm2"] = ((W,), "small")
        if f["kind"] == "dense":
            out[f"l{i}.mlp.up"] = ((f["ff"], W), "matrix")
            out[f"l{i}.mlp.down"] = ((W, f["ff"]), "matrix")
            continue
        ff = f["expert"]["ff"]
        for e in range(f["router"]["experts"]):
            out[f"l{i}.mlp.e{e}.gate"] = ((ff, W), "matrix")
            out[f"l{i}.mlp.e{e}.up"] = ((ff, W), "matrix")
            out[f"l{i}.mlp.e{e}.down"] = ((W, ff), "matrix")
        out[f"l{i}.mlp.router"] = ((f["router"]["experts"], W), "router")
    out["final.norm"] = ((W,), "small")
    out["head"] = ((cfg["vocab"], W), "matrix")
    return out


def random_weights(cfg, seed=0, **sizes):
    """float32 weights, each rounded to bfloat16 values so that every engine dtype holds the same numbers."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, (shape, kind) in tensor_shapes(cfg, **sizes).items():
        r = torch.randn(shape, generator=g)
        if kind == "embed":
            t = r * 0.7
        elif kind == "matrix":
            t = r / math.sqrt(shape[-1])
        elif kind == "router":
            t = r * (2.0 / math.sqrt(shape[-1]))
        elif kind == "norm":
            t = 1.0 + 0.2 * r
        elif kind == "mu":
            t = torch.rand(shape, generator=g)
        elif kind == "conv":
            t = r / math.sqrt(shape[-1])
        elif kind == "rel":
            t = r
        elif kind == "a_log":
            t = 0.5 * r  # decays of about exp(-dt)
        elif kind == "dt_bias":
            t = -2.0 + r  # steps of about 0.1, so that a state lives for tens of tokens
        elif kind == "w0":
            t = -3.0 + 1.5 * r  # decays of about 0.95, some near 1, some near 0.3
        else:
            t = 0.2 * r
        w[name] = t.to(torch.bfloat16).float()
    return w
