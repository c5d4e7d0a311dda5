"""Plain float64 restatement of the Tibelix design, one function per mechanism, numpy only.

Test infrastructure: nothing under ntransformer_b200/ imports it and it shares no code with the product path.  It keeps no cache and
no state: every function sees the whole sequence (the matrix memory is a loop over time), so the product's cache, state hand-over and
schedules are checked against something that cannot have the same fault.  `store`, where a function takes it, is applied to whatever the product
keeps in 16 bits (cache rows, and the per-head keys and values it expands latent rows to): None keeps everything in float64.

Notation.  X is [T, width]; weights are [out, in] and applied as x @ W.T.  `cfg` is the parsed config.json, `P` maps tensor names to
float64 arrays.
"""
from __future__ import annotations

import math

import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_zero(x, w, eps):
    """Gain stored around zero."""
    return rms(x, eps) * (1.0 + w)


def norm_plain(x, w, eps):
    return rms(x, eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


# ---------------------------------------------------------------- attention
def query_temperature(pos, coef, every):
    """1 + coef ln(floor((p + 1) / every) + 1)."""
    return np.array([1.0 + coef * math.log(math.floor((int(p) + 1) / every) + 1) for p in pos])


def slopes(H):
    return np.array([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)])


def causal(T):
    return np.tril(np.ones((T, T), dtype=bool))


def sink_softmax(s, mask):
    """exp(s) / (1 + sum exp(s)) over the visible keys."""
    s = np.where(mask, s, -np.inf)
    m = np.maximum(s.max(axis=-1, keepdims=True), 0.0)
    e = np.exp(s - m)
    return e / (np.exp(-m) + e.sum(axis=-1, keepdims=True))


def softmax_rows(s, mask):
    s = np.where(mask, s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def kept(x, store):
    return store(x) if store else x


def attention_kv(h, P, p, m, eps, store=None):
    """Keys [T, G, dim] (unit root mean square per head) and values [T, G, vdim]."""
    T, G = h.shape[0], m["kv_heads"]
    return kept(rms((h @ P[p + "k"].T).reshape(T, G, m["dim"]), eps), store), kept((h @ P[p + "v"].T).reshape(T, G, m["vdim"]), store)


def biased_attention(q, k, v, scale, slope):
    """q [T, H, D] against k [T, G, D], v [T, G, V]: scores minus slope times the distance, one more 1 in the denominator."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    dist = np.arange(T)[:, None] - np.arange(T)[None, :]
    out = np.zeros((T, H, v.shape[2]))
    for x in range(H):
        g = x // (H // G)
        s = q[:, x] @ k[:, g].T * scale - slope[x] * dist
        out[:, x] = sink_softmax(s, causal(T)) @ v[:, g]
    return out


def attention(h, P, p, m, eps, kv):
    T, H = h.shape[0], m["heads"]
    q = rms((h @ P[p + "q"].T).reshape(T, H, m["dim"]), eps)
    t = m.get("q_temp")
    if t:
        q = q * query_temperature(range(T), t["coef"], t["every"])[:, None, None]
    o = biased_attention(q, kv[0], kv[1], m["scale"], slopes(H)) * sigmoid(h @ P[p + "g"].T)[:, :, None]
    return o.reshape(T, -1) @ P[p + "o"].T


# ---------------------------------------------------------------- latent attention
def blended_frequencies(dims, base, scaling):
    """Angular frequency of every pair, and what cos and sin are multiplied by."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return np.array(f), 1.0

    def turn(t):
        return dims * math.log(scaling["original"] / (2 * math.pi * t)) / (2 * math.log(base))

    lo, hi = max(math.floor(turn(scaling["fast"])), 0), min(math.ceil(turn(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / scaling["factor"] * r + fi * (1.0 - r))
    return np.array(out), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_pairs(v, pos, rot):
    """v [T, ..., d]: channel 2i turns with channel 2i + 1 by pos * f_i; channels past rot.dims pass."""
    if not rot or rot["dims"] == 0:
        return v.copy()
    out, n = v.copy(), rot["dims"]
    f, mag = blended_frequencies(n, rot["base"], rot.get("scaling"))
    a = np.asarray(pos, dtype=np.float64).reshape((-1,) + (1,) * (v.ndim - 1)) * f
    c, s = np.cos(a) * mag, np.sin(a) * mag
    x, y = v[..., 0:n:2], v[..., 1:n:2]
    out[..., 0:n:2] = x * c - y * s
    out[..., 1:n:2] = y * c + x * s
    return out


def latent_attention(h, P, p, m, eps, store=None, expanded=False):
    T = h.shape[0]
    H, D, R, V, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    cq = norm_plain(h @ P[p + "dq"].T, P[p + "dq.norm"], eps)
    q = (cq @ P[p + "uq"].T).reshape(T, H, D + R)
    qn, qr = q[:, :, :D], rotate_pairs(q[:, :, D:], pos, m.get("rot"))
    d = h @ P[p + "dkv"].T
    c, kr = kept(norm_plain(d[:, :r], P[p + "dkv.norm"], eps), store), kept(rotate_pairs(d[:, r:], pos, m.get("rot")), store)
    kn, v = (c @ P[p + "uk"].T).reshape(T, H, D), (c @ P[p + "uv"].T).reshape(T, H, V)
    if expanded:
        kn, v = kept(kn, store), kept(v, store)
    out = np.zeros((T, H, V))
    for x in range(H):
        s = (qn[:, x] @ kn[:, x].T + qr[:, x] @ kr.T) * m["scale"]
        out[:, x] = softmax_rows(s, causal(T)) @ v[:, x]
    return (out.reshape(T, H * V) * sigmoid(h @ P[p + "g"].T)) @ P[p + "o"].T


# ---------------------------------------------------------------- matrix memory
def mlstm_gates(zi, zf, cap):
    """Log input gate and log forget gate from their pre-activations (bias added)."""
    return soft_cap(zi, cap), log_sigmoid(soft_cap(zf, cap))


def mlstm_memory(q, k, v, i, f):
    """q, k [T, H, D] (q scaled), v [T, H, V], log gates i, f [T, H] -> o [T, H, V] and the final (S, n, m)."""
    T, H, D = q.shape
    S, n, m = np.zeros((H, D, v.shape[2])), np.zeros((H, D)), np.zeros(H)
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        mt = np.maximum(f[t] + m, i[t])
        a, b = np.exp(f[t] + m - mt), np.exp(i[t] - mt)
        S = a[:, None, None] * S + b[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = a[:, None] * n + b[:, None] * k[t]
        m = mt
        den = np.maximum(np.abs(np.einsum("hd,hd->h", n, q[t])), np.exp(-m)) + 1e-6
        o[t] = np.einsum("hdv,hd->hv", S, q[t]) / den[:, None]
    return o, (S, n, m)


def mlstm(h, P, p, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = (h @ P[p + "q"].T).reshape(T, H, D) * D ** -0.5, (h @ P[p + "k"].T).reshape(T, H, D)
    v = (h @ P[p + "v"].T).reshape(T, H, V)
    i, f = mlstm_gates(h @ P[p + "i"].T + P[p + "i.b"], h @ P[p + "f"].T + P[p + "f.b"], m["gate_cap"])
    o = rms(mlstm_memory(q, k, v, i, f)[0], eps).reshape(T, H * V)
    return (o * P[p + "norm"] * sigmoid(h @ P[p + "g"].T)) @ P[p + "o"].T


# ---------------------------------------------------------------- feed-forward
def dense_ff(h, P, p):
    return np.maximum(h @ P[p + "up"].T, 0.0) ** 2 @ P[p + "down"].T


def gated_unit(h, P, p):
    return (silu(h @ P[p + "gate"].T) * (h @ P[p + "up"].T)) @ P[p + "down"].T


def route(h, router, top, groups=None):
    """Softmax over all experts; groups score their best expert and only the best `keep` groups can be chosen from; the chosen shares sum to one."""
    z = h @ router.T
    e = np.exp(z - z.max(axis=1, keepdims=True))
    s = e / e.sum(axis=1, keepdims=True)
    c = s.copy()
    if groups:
        g = s.reshape(len(s), groups["count"], -1)
        best = np.argsort(-g.max(axis=2), axis=1, kind="stable")[:, :groups["keep"]]
        ok = np.zeros(g.shape[:2], dtype=bool)
        np.put_along_axis(ok, best, True, axis=1)
        c = np.where(ok[:, :, None], g, -1.0).reshape(s.shape)
    sel = np.argsort(-c, axis=1, kind="stable")[:, :top]
    w = np.take_along_axis(s, sel, axis=1)
    return sel, w / (w.sum(axis=1, keepdims=True) + 1e-20)


def moe_ff(h, P, p, mlp):
    rt = mlp["router"]
    sel, wt = route(h, P[p + "router"], rt["top"], rt.get("groups"))
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(sel[t], wt[t]):
            y[t] += w * gated_unit(h[t:t + 1], P, p + "e%d." % e)[0]
    return y + gated_unit(h, P, p + "shared.") if mlp.get("shared") else y


# ---------------------------------------------------------------- model
def layers(cfg, P, tokens, store=None, expanded=False):
    """The embedding output, then the residual after every layer."""
    eps = cfg["norm"]["eps"]
    x = P["embed"][np.asarray(tokens)]
    out, kv = [x], {}
    for i, e in enumerate(cfg["layers"]):
        p, m = "l%d." % i, e["mixer"]
        h = norm_zero(x, P[p + "norm1"], eps)
        if e["type"] == "attention":
            if "kv_from" not in m:
                kv[i] = attention_kv(h, P, p + "mix.", m, eps, store)
            y = attention(h, P, p + "mix.", m, eps, kv[m.get("kv_from", i)])
        elif e["type"] == "latent_attention":
            y = latent_attention(h, P, p + "mix.", m, eps, store, expanded)
        else:
            y = mlstm(h, P, p + "mix.", m, eps)
        x = x + norm_zero(y, P[p + "norm1b"], eps)
        f = e.get("mlp")
        if f:
            h = norm_zero(x, P[p + "norm2"], eps)
            y = dense_ff(h, P, p + "mlp.") if f["kind"] == "dense" else moe_ff(h, P, p + "mlp.", f)
            x = x + norm_zero(y, P[p + "norm2b"], eps)
        out.append(x)
    return out


def forward(cfg, P, tokens, store=None, expanded=False):
    return norm_zero(layers(cfg, P, tokens, store, expanded)[-1], P["final.norm"], cfg["norm"]["eps"]) @ P["embed"].T


# ---------------------------------------------------------------- random models
def bf16_grid(a):
    """Nearest values that BF16 can hold."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32).astype(np.float64)


def random_model(rng, pattern=("attention", "latent_attention", "mlstm", "attention"), mlp=("dense", "moe", None, "moe"), kv_from=None, width=36, vocab=61, eps=1e-5,
                 heads=6, kv_heads=3, dim=10, vdim=7, scale=None, temp=(0.7, 5), l_heads=3, l_dim=9, rot_dim=6, l_vdim=5, q_rank=13, kv_rank=11, rot_dims=None,
                 rot_base=500.0, scaling=(4.0, 40, 8.0, 1.0), l_scale=None, m_heads=2, m_dim=9, m_vdim=11, cap=8.0, ff=23, experts=6, top=2, groups=(3, 2), eff=12,
                 shared=17, gain=1.0):
    """A small configuration and random weights on the BF16 grid.  mlp: feed-forward kind per layer ("dense", "moe", None); kv_from: {layer: earlier
    attention layer}; temp, scaling, groups: None switches the mechanism off; shared 0: no shared expert."""
    kv_from = kv_from or {}
    lay = []
    for i, typ in enumerate(pattern):
        if typ == "attention":
            m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale else dim ** -0.5}
            if temp:
                m["q_temp"] = {"coef": temp[0], "every": temp[1]}
            if i in kv_from:
                m["kv_from"] = kv_from[i]
        elif typ == "latent_attention":
            m = {"heads": l_heads, "dim": l_dim, "rot_dim": rot_dim, "vdim": l_vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                 "scale": l_scale if l_scale else (l_dim + rot_dim) ** -0.5, "rot": {"base": rot_base, "dims": rot_dim if rot_dims is None else rot_dims}}
            if scaling:
                m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
        else:
            m = {"heads": m_heads, "dim": m_dim, "vdim": m_vdim, "gate_cap": cap}
        k = mlp[i % len(mlp)]
        if k == "dense":
            f = {"kind": "dense", "ff": ff}
        elif k == "moe":
            f = {"kind": "moe", "expert": {"ff": eff}, "router": {"experts": experts, "top": top}}
            if groups:
                f["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
            if shared:
                f["shared"] = {"ff": shared}
        else:
            f = None
        lay.append({"type": typ, "mixer": m, "mlp": f})
    cfg = {"architecture": "Tibelix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": lay}

    def mat(r, c, g=1.0):
        return rng.standard_normal((r, c)) * gain * g * c ** -0.5

    def vec(n, mean=0.0, std=0.2):
        return mean + std * rng.standard_normal(n)

    P = {"embed": rng.standard_normal((vocab, width)), "final.norm": vec(width)}
    for i, e in enumerate(lay):
        p, m = "l%d." % i, e["mixer"]
        q = p + "mix."
        P[p + "norm1"], P[p + "norm1b"] = vec(width), vec(width)
        H, D, V = m["heads"], m["dim"], m["vdim"]
        if e["type"] == "attention":
            P[q + "q"] = mat(H * D, width)
            if "kv_from" not in m:
                P[q + "k"], P[q + "v"] = mat(m["kv_heads"] * D, width), mat(m["kv_heads"] * V, width)
            P[q + "g"] = mat(H, width)
        elif e["type"] == "latent_attention":
            R, r = m["rot_dim"], m["kv_rank"]
            P[q + "dq"], P[q + "dq.norm"], P[q + "uq"] = mat(m["q_rank"], width), vec(m["q_rank"], 1.0), mat(H * (D + R), m["q_rank"])
            P[q + "dkv"], P[q + "dkv.norm"] = mat(r + R, width), vec(r, 1.0)
            P[q + "uk"], P[q + "uv"], P[q + "g"] = mat(H * D, r), mat(H * V, r), mat(H * V, width)
        else:
            P[q + "q"], P[q + "k"], P[q + "v"], P[q + "g"] = mat(H * D, width), mat(H * D, width), mat(H * V, width), mat(H * V, width)
            P[q + "i"], P[q + "f"] = mat(H, width, 2.0), mat(H, width, 2.0)
            P[q + "i.b"], P[q + "f.b"] = vec(H, -1.0, 1.0), vec(H, 3.0, 1.0)
            P[q + "norm"] = vec(H * V, 1.0)
        P[q + "o"] = mat(width, H * V)
        f = e["mlp"]
        if f:
            P[p + "norm2"], P[p + "norm2b"] = vec(width), vec(width)
        if f and f["kind"] == "dense":
            P[p + "mlp.up"], P[p + "mlp.down"] = mat(f["ff"], width), mat(width, f["ff"])
        elif f:
            P[p + "mlp.router"] = mat(f["router"]["experts"], width, 2.0)
            for n in ["e%d" % x for x in range(f["router"]["experts"])] + (["shared"] if f.get("shared") else []):
                w = f["shared"]["ff"] if n == "shared" else f["expert"]["ff"]
                for s, (r, c) in (("gate", (w, width)), ("up", (w, width)), ("down", (width, w))):
                    P[p + "mlp." + n + "." + s] = mat(r, c)
    return cfg, {k: bf16_grid(a) for k, a in P.items()}
