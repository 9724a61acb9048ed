"""The Mafarax decoder restated plainly: one slow function per mechanism, whole sequences at once, any float
dtype (the tests run it in 64-bit on the weights as given).  It shares no code with the engine.

Notation: n tokens, positions 0 .. n-1; x [n, width]; a linear map is `x @ W.T` with W [out, in].
"""

from __future__ import annotations

import math

import torch


# ---------------------------------------------------------------------------------------------------------
# norms, rotation
# ---------------------------------------------------------------------------------------------------------
def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def dynamic_tanh(x, w, name):
    """tanh(alpha x) * weight + b: no statistics of the row at all."""
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def rotate_halves(v, positions, dims, base, factor=1.0):
    """v [..., n, d]: (i, i + dims / 2), i < dims / 2, turn by position * base^(-2i / dims) / factor; the rest stays."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = (torch.pow(torch.tensor(float(base), dtype=torch.float64), -2.0 * i / dims) / factor).to(v.dtype)
    a = positions.to(v.dtype)[:, None] * f[None, :]
    c, s = torch.cos(a), torch.sin(a)
    h = dims // 2
    p, r = v[..., :h], v[..., h:dims]
    out = v.clone()
    out[..., :h] = p * c - r * s
    out[..., h:dims] = r * c + p * s
    return out


# ---------------------------------------------------------------------------------------------------------
# the left mixer: attention inside chunks
# ---------------------------------------------------------------------------------------------------------
def chunked_attention_core(q, k, v, scale, size):
    """q [H, n, d], k [G, n, d], v [G, n, dv] -> [n, H * dv].  Query i sees the keys j <= i of its own stretch of
    `size` positions (None: every j <= i); stretches are counted from position 0."""
    H, n, _ = q.shape
    G, dv = k.shape[0], v.shape[-1]
    rep = H // G
    out = torch.zeros(n, H, dv, dtype=q.dtype)
    for i in range(n):
        lo = 0 if size is None else (i // size) * size
        for h in range(H):
            g = h // rep
            p = torch.softmax((k[g, lo:i + 1] @ q[h, i]) * scale, 0)
            out[i, h] = p @ v[g, lo:i + 1]
    return out.reshape(n, H * dv)


def left_mixer(h, m, w, pre):
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(n)

    def proj(name, heads, size):
        return (h @ w[pre + name].T + w[pre + name + ".b"]).reshape(n, heads, size).transpose(0, 1)

    q, k, v = proj("q", H, d), proj("k", G, d), proj("v", G, dv)
    rot = m.get("rot")
    if rot:
        factor = (rot.get("scaling") or {}).get("factor", 1.0)
        q = rotate_halves(q, pos, rot["dims"], rot["base"], factor)
        k = rotate_halves(k, pos, rot["dims"], rot["base"], factor)
    size = m["mask"]["size"] if m.get("mask") else None
    a = chunked_attention_core(q, k, v, m["scale"], size)
    return a @ w[pre + "o"].T + w[pre + "o.b"]


# ---------------------------------------------------------------------------------------------------------
# the right mixer: a state-space recurrence with a scalar decay per head
# ---------------------------------------------------------------------------------------------------------
def causal_conv_silu(u, taps_w, bias):
    """u [n, channels]; taps_w [channels, taps], the last column meets the current token; zeros before the start."""
    n, taps = u.shape[0], taps_w.shape[1]
    y = bias[None, :].repeat(n, 1)
    for j in range(taps):
        back = taps - 1 - j
        if back < n:
            y[back:] = y[back:] + u[:n - back] * taps_w[:, j]
    return y * torch.sigmoid(y)


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


def gate_then_group_norm(y, z, parts, w, eps):
    g = y * (z * torch.sigmoid(z))
    n, inner = g.shape
    p = g.reshape(n, parts, inner // parts)
    p = p / torch.sqrt((p * p).mean(-1, keepdim=True) + eps)
    return p.reshape(n, inner) * w


def right_mixer(h, m, w, pre, eps):
    n = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    u = h @ w[pre + "in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = causal_conv_silu(xbc, w[pre + "conv"], w[pre + "conv.b"])
    x = xbc[:, :inner].reshape(n, H, P)
    B = xbc[:, inner:inner + G * N].reshape(n, G, N)
    C = xbc[:, inner + G * N:].reshape(n, G, N)
    dt = torch.nn.functional.softplus(dt + w[pre + "dt_bias"], threshold=200.0)
    y = state_space_core(x, B, C, dt, w[pre + "A_log"], w[pre + "D"]).reshape(n, inner)
    return gate_then_group_norm(y, z, m["norm_groups"], w[pre + "norm"], eps) @ w[pre + "o"].T


def parallel_mixer(h, m, w, pre, eps):
    left = left_mixer(h, m["left"], w, pre + "left.")
    right = right_mixer(h, m["right"], w, pre + "right.", eps)
    return 0.5 * (rms_norm(left, w[pre + "left.out"], eps) + rms_norm(right, w[pre + "right.out"], eps))


# ---------------------------------------------------------------------------------------------------------
# feed-forward
# ---------------------------------------------------------------------------------------------------------
def expert(h, w, pre):
    return torch.relu(h @ w[pre + "up"].T) ** 2 @ w[pre + "down"].T


def route(h, w, pre, r):
    """(chosen [n, top], their weights [n, top]).  Ties go to the lower index, groups as well as experts."""
    E, top = r["experts"], r["top"]
    s = torch.sigmoid(h @ w[pre + "router"].T)
    chosen = torch.zeros(h.shape[0], top, dtype=torch.long)
    gr = r.get("groups") or dict(count=1, keep=1)
    per = E // gr["count"]
    for t in range(h.shape[0]):
        allowed = list(range(E))
        if gr["keep"] < gr["count"]:
            rank = [sum(sorted((float(s[t, e]) for e in range(g * per, (g + 1) * per)), reverse=True)[:2])
                    for g in range(gr["count"])]
            best = sorted(range(gr["count"]), key=lambda g: (-rank[g], g))[:gr["keep"]]
            allowed = [e for e in range(E) if e // per in best]
        order = sorted(allowed, key=lambda e: (-float(s[t, e]), e))
        chosen[t] = torch.tensor(order[:top])
    return chosen, torch.gather(s, 1, chosen) * r["scale"]


def routed_ff(h, f, w, pre):
    chosen, weight = route(h, w, pre, f["router"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(chosen.shape[1]):
            y[t] += weight[t, j] * expert(h[t:t + 1], w, f"{pre}e{int(chosen[t, j])}.")[0]
    if f.get("shared"):
        y = y + expert(h, w, pre + "shared.")
    return y


# ---------------------------------------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------------------------------------
def layer(x, i, cfg, w):
    L, eps, pre = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}."
    x = x + parallel_mixer(dynamic_tanh(x, w, pre + "norm1"), L["mixer"], w, pre + "mix.", eps)
    if L.get("mlp") is not None:
        x = x + routed_ff(dynamic_tanh(x, w, pre + "norm2"), L["mlp"], w, pre + "mlp.")
    return x


def forward(cfg, w, ids, return_layers: bool = False):
    """Logits [n, vocab] of one sequence (and the stream after every layer, if asked)."""
    x = w["embed"][torch.as_tensor(ids, dtype=torch.long)]
    seen = []
    for i in range(len(cfg["layers"])):
        x = layer(x, i, cfg, w)
        seen.append(x)
    logits = (dynamic_tanh(x, w, "final.norm") @ w["head"].T) * cfg["logit_scale"]
    return (logits, torch.stack(seen)) if return_layers else logits


# ---------------------------------------------------------------------------------------------------------
# shapes and random weights
# ---------------------------------------------------------------------------------------------------------
def tensor_shapes(cfg):
    """{name: (shape, kind)}; kind: "matrix", "router", "norm" (near 1), "small" (near 0), "alpha" (a positive
    slope), "conv", "a_log", "dt_bias"."""
    W, out = cfg["width"], {}

    def norm(name):
        out[name] = ((W,), "norm")
        out[name + ".b"] = ((W,), "small")
        out[name + ".alpha"] = ((), "alpha")

    out["embed"] = ((cfg["vocab"], W), "embed")
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        norm(p + "norm1")
        a, pl = m["left"], p + "mix.left."
        H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        for name, rows, cols in (("q", H * d, W), ("k", G * d, W), ("v", G * dv, W), ("o", W, H * dv)):
            out[pl + name] = ((rows, cols), "matrix")
            out[pl + name + ".b"] = ((rows,), "small")
        s, pr = m["right"], p + "mix.right."
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
        if f is not None:
            norm(p + "norm2")
            ff = f["expert"]["ff"]
            for e in range(f["router"]["experts"]):
                out[f"{p}mlp.e{e}.up"] = ((ff, W), "matrix")
                out[f"{p}mlp.e{e}.down"] = ((W, ff), "matrix")
            out[p + "mlp.router"] = ((f["router"]["experts"], W), "router")
            if f.get("shared"):
                out[p + "mlp.shared.up"] = ((f["shared"]["ff"], W), "matrix")
                out[p + "mlp.shared.down"] = ((W, f["shared"]["ff"]), "matrix")
    norm("final.norm")
    out["head"] = ((cfg["vocab"], W), "matrix")
    return out


def random_weights(cfg, seed=0):
    """float32 weights, each rounded to bfloat16 values so that every engine dtype holds the same numbers."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, (shape, kind) in tensor_shapes(cfg).items():
        r = torch.randn(shape, generator=g)
        if kind == "embed":
            t = r
        elif kind == "matrix":
            t = r / math.sqrt(shape[-1])
        elif kind == "router":
            t = r * (2.0 / math.sqrt(shape[-1]))
        elif kind == "norm":
            t = 1.0 + 0.2 * r
        elif kind == "alpha":
            t = 0.5 + 0.3 * torch.rand(shape, generator=g)
        elif kind == "conv":
            t = r / math.sqrt(shape[-1])
        elif kind == "a_log":
            t = 0.5 * r  # decays of about exp(-dt)
        elif kind == "dt_bias":
            t = -2.0 + r  # steps of about 0.1, so that a state lives for tens of tokens
        else:
            t = 0.2 * r
        w[name] = t.to(torch.bfloat16).float()
    return w
