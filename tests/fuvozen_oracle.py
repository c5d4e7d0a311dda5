"""Plain float64 restatement of the Fuvozen design, one function per mechanism, numpy only.

Test infrastructure: nothing under ntransformer_b200/ imports it and it shares no code with the product path.  It keeps no cache and
no state: every function sees the whole sequence (the recurrence is a loop over time), so the product's cache, state hand-over and
schedules are checked against something that cannot have the same fault.

Notation.  X is [T, width]; weights are [out, in] and applied as x @ W.T.  `cfg` is the parsed config.json, `P` maps tensor names to
float64 arrays.
"""
from __future__ import annotations

import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_plain(x, w, eps):
    return rms(x, eps) * w


def norm_groups(x, w, groups, eps):
    """Every one of `groups` equal runs of channels has its own root mean square; one gain over the whole vector."""
    T, W = x.shape
    return rms(x.reshape(T, groups, W // groups), eps).reshape(T, W) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def xielu(z, p, q):
    """z > 0: softplus(p) z^2 + z / 2;  z <= 0: (1/2 + softplus(q)) (e^z - 1 - z) + z / 2."""
    neg = np.minimum(z, 0.0)
    return np.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (np.expm1(neg) - neg)) + 0.5 * z


def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the second table for every position; the first token of a sequence reads the row behind the hashed ones."""
    rows = [buckets]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((int(prev) * mul_prev + int(cur) * mul_cur) % buckets)
    return np.asarray(rows[:len(tokens)], dtype=np.int64)


def embedding(cfg, P, tokens):
    x = P["embed"][np.asarray(tokens)]
    b = cfg["embedding"]["bigram"]
    return x + P["bigram"][bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"])]


def depth_average(Xs, w):
    """sum_j w[j] X_j over everything the depth has produced so far."""
    return sum(wj * Xj for wj, Xj in zip(w, Xs))


def rotate_pairs(v, pos, dims, base):
    """v [T, ..., d]: channel 2i turns with channel 2i + 1 by pos * base^(-2i / dims), i < dims / 2; the rest pass."""
    out = v.copy()
    f = base ** (-2.0 * np.arange(dims // 2) / max(dims, 1))
    a = np.asarray(pos, dtype=np.float64).reshape((-1,) + (1,) * (v.ndim - 1)) * f
    c, s = np.cos(a), np.sin(a)
    u, w = v[..., 0:dims:2], v[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - w * s
    out[..., 1:dims:2] = w * c + u * s
    return out


def window_mask(T, size):
    """[i, j]: 0 <= i - j < size (size None: every j <= i)."""
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & ((d < size) if size else True)


def softmax_rows(s, mask):
    s = np.where(mask, s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def latent_kv(h, P, p, m, eps, pos):
    """The normed latent [T, kv_rank] and the rotated key part [T, rot_dim] that all heads share."""
    r = m["kv_rank"]
    d = h @ P[p + "dkv"].T
    return norm_plain(d[:, :r], P[p + "dkv.norm"], eps), rotate_pairs(d[:, r:], pos, m["rot"]["dims"], m["rot"]["base"])


def latent_attention(h, P, p, m, eps):
    T = h.shape[0]
    H, D, R, V = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    pos = np.arange(T)
    c, kr = latent_kv(h, P, p, m, eps, pos)
    q = (h @ P[p + "q"].T).reshape(T, H, D + R)
    qn, qr = q[:, :, :D], rotate_pairs(q[:, :, D:], pos, m["rot"]["dims"], m["rot"]["base"])
    kn = (c @ P[p + "uk"].T).reshape(T, H, D)
    v = (c @ P[p + "uv"].T).reshape(T, H, V)
    mask = window_mask(T, (m.get("mask") or {}).get("size"))
    out = np.zeros((T, H, V))
    for g in range(H):
        s = (qn[:, g] @ kn[:, g].T + qr[:, g] @ kr.T) * m["scale"]
        out[:, g] = softmax_rows(s, mask) @ v[:, g]
    return out.reshape(T, H * V) @ P[p + "o"].T


def shifted(h):
    """The previous token's row; zeros in front of the first."""
    return np.concatenate([np.zeros((1, h.shape[1])), h[:-1]], axis=0)


def wkv_recurrence(r, k, v, w, u):
    """r, k, w [T, H, D], v [T, H, V], u [H, D]: o_t = (S + (u k_t) v_t^T)^T r_t, then S <- w_t S + k_t v_t^T per head, S [D, V] from zero."""
    T, H, D = r.shape
    S = np.zeros((H, D, v.shape[2]))
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hd,hdv->hv", r[t], S + u[:, :, None] * kv)
        S = w[t][:, :, None] * S + kv
    return o


def wkv(h, P, p, m, eps):
    T = h.shape[0]
    H, D = m["heads"], m["dim"]
    d = shifted(h) - h
    mix = {s: h + d * P[p + "mu." + s] for s in "rkvgw"}
    r, k, v = ((mix[s] @ P[p + s].T).reshape(T, H, D) for s in "rkv")
    gate = silu(mix["g"] @ P[p + "g"].T)
    w = np.exp(-np.exp(np.tanh(mix["w"] @ P[p + "w1"].T) @ P[p + "w2"].T + P[p + "w0"])).reshape(T, H, D)
    o = rms(wkv_recurrence(r, k, v, w, P[p + "u"]), eps).reshape(T, H * D)
    return (o * P[p + "norm"] * gate) @ P[p + "o"].T


def dense_ff(h, P, p):
    a = P[p + "act"]
    return xielu(h @ P[p + "up"].T, a[0], a[1]) @ P[p + "down"].T


def gated_unit(h, P, p):
    return (silu(h @ P[p + "gate"].T) * (h @ P[p + "up"].T)) @ P[p + "down"].T


def route(h, router, top, scale):
    """Softmax over all experts; the `top` largest keep their share times `scale` (not renormalized)."""
    z = h @ router.T
    e = np.exp(z - z.max(axis=1, keepdims=True))
    s = e / e.sum(axis=1, keepdims=True)
    sel = np.argsort(-s, axis=1, kind="stable")[:, :top]
    return sel, np.take_along_axis(s, sel, axis=1) * scale


def moe_ff(h, P, p, mlp):
    rt = mlp["router"]
    sel, wt = route(h, P[p + "router"], rt["top"], rt["scale"])
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(sel[t], wt[t]):
            y[t] += w * gated_unit(h[t:t + 1], P, p + "e%d." % e)[0]
    return y + gated_unit(h, P, p + "shared.") if mlp.get("shared") else y


def layers(cfg, P, tokens):
    """The embedding output, then the stream after every layer (behind the average over depth)."""
    eps, G = cfg["norm"]["eps"], cfg["norm"]["groups"]
    x = embedding(cfg, P, tokens)
    Xs, out = [x], [x]
    for i, e in enumerate(cfg["layers"]):
        p = "l%d." % i
        h = norm_groups(x, P[p + "norm1"], G, eps)
        mix = wkv if e["type"] == "wkv" else latent_attention
        y = mix(h, P, p + "mix.", e["mixer"], eps)
        f = e.get("mlp")
        if f:
            y = y + (dense_ff(h, P, p + "mlp.") if f["kind"] == "dense" else moe_ff(h, P, p + "mlp.", f))
        Xs.append(x + y)
        x = depth_average(Xs, P[p + "dwa"])
        out.append(x)
    return out


def forward(cfg, P, tokens):
    x = layers(cfg, P, tokens)[-1]
    return norm_groups(x, P["final.norm"], cfg["norm"]["groups"], cfg["norm"]["eps"]) @ P["embed"].T


# ---------------------------------------------------------------- random models
def bf16_grid(a):
    """Nearest values that BF16 can hold."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32).astype(np.float64)


def random_model(rng, pattern=("wkv", "latent_attention", "wkv", "latent_attention"), mlp=("dense", "moe", "moe", "dense"), width=36, vocab=61, groups=3,
                 eps=1e-5, buckets=97, mul_prev=13, mul_cur=7, heads=3, dim=10, rot_dim=6, vdim=7, kv_rank=11, window=9, rot_base=500.0, scale=None,
                 w_heads=2, w_dim=9, rank=5, ff=23, experts=5, top=2, eff=12, shared=17, router_scale=1.7, gain=1.0):
    """A small configuration and random weights on the BF16 grid.  mlp: feed-forward kind per layer ("dense", "moe", None)."""
    lay = []
    for i, typ in enumerate(pattern):
        if typ == "wkv":
            m = {"heads": w_heads, "dim": w_dim, "decay_rank": rank}
        else:
            m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale if scale else (dim + rot_dim) ** -0.5,
                 "rot": {"base": rot_base, "dims": rot_dim}}
            if window:
                m["mask"] = {"size": window}
        k = mlp[i % len(mlp)]
        if k == "dense":
            f = {"kind": "dense", "ff": ff}
        elif k == "moe":
            f = {"kind": "moe", "expert": {"ff": eff}, "router": {"experts": experts, "top": top, "scale": router_scale}}
            if shared:
                f["shared"] = {"ff": shared}
        else:
            f = None
        lay.append({"type": typ, "mixer": m, "mlp": f})
    cfg = {"architecture": "Fuvozen", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups},
           "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}, "layers": lay}

    def mat(r, c):
        return rng.standard_normal((r, c)) * gain * c ** -0.5

    def vec(n, mean=1.0, std=0.2):
        return mean + std * rng.standard_normal(n)

    P = {"embed": rng.standard_normal((vocab, width)), "bigram": 0.7 * rng.standard_normal((buckets + 1, width)), "final.norm": vec(width)}
    for i, e in enumerate(lay):
        p, m = "l%d." % i, e["mixer"]
        P[p + "norm1"] = vec(width)
        q = p + "mix."
        if e["type"] == "wkv":
            n = m["heads"] * m["dim"]
            for s in "rkvgw":
                P[q + "mu." + s] = rng.uniform(0.0, 1.0, width)
            for s in "rkvg":
                P[q + s] = mat(n, width)
            P[q + "w1"], P[q + "w2"] = mat(rank, width), mat(n, rank)
            P[q + "w0"] = rng.uniform(-4.0, 0.5, n)
            P[q + "u"] = rng.standard_normal((m["heads"], m["dim"]))
            P[q + "norm"] = vec(n)
            P[q + "o"] = mat(width, n)
        else:
            P[q + "q"] = mat(m["heads"] * (m["dim"] + m["rot_dim"]), width)
            P[q + "dkv"] = mat(m["kv_rank"] + m["rot_dim"], width)
            P[q + "dkv.norm"] = vec(m["kv_rank"])
            P[q + "uk"] = mat(m["heads"] * m["dim"], m["kv_rank"])
            P[q + "uv"] = mat(m["heads"] * m["vdim"], m["kv_rank"])
            P[q + "o"] = mat(width, m["heads"] * m["vdim"])
        f = e["mlp"]
        if f and f["kind"] == "dense":
            P[p + "mlp.up"], P[p + "mlp.down"] = mat(f["ff"], width), mat(width, f["ff"])
            P[p + "mlp.act"] = rng.uniform(-1.0, 0.5, 2)
        elif f:
            P[p + "mlp.router"] = 2.0 * mat(f["router"]["experts"], width)
            names = ["e%d" % x for x in range(f["router"]["experts"])] + (["shared"] if f.get("shared") else [])
            for n in names:
                w = f["shared"]["ff"] if n == "shared" else f["expert"]["ff"]
                for s, (r, c) in (("gate", (w, width)), ("up", (w, width)), ("down", (width, w))):
                    P[p + "mlp." + n + "." + s] = mat(r, c)
        P[p + "dwa"] = np.concatenate([rng.uniform(-0.2, 0.3, i + 1), [1.0 + 0.2 * rng.standard_normal()]])
    return cfg, {k: bf16_grid(a) for k, a in P.items()}
