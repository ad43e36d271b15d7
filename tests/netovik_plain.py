"""Plain, slow float64 statement of the Netovik design: one function per mechanism, whole sequences, no cache and no batch.

A model is (config dict as it stands in config.json, {tensor name: float64 array}).  Nothing here comes from the package:
the tests compare the engine with these functions."""
import math

import numpy as np

from pavatar_plain import sigmoid  # noqa: F401  (plain statements as well)
from sokirax_plain import silu, softmax, unit_rms  # noqa: F401
from vefilix_plain import bf16, write_model  # noqa: F401


def grouped_norm(x, w, groups, eps):
    """Every one of ``groups`` consecutive parts of a row over its own root mean square, the row then times w."""
    parts = x.reshape(*x.shape[:-1], groups, -1)
    return (parts / np.sqrt((parts * parts).mean(-1, keepdims=True) + eps)).reshape(x.shape) * w


def depth_average(streams, c):
    """streams: the embedding and every layer's result so far."""
    return sum(c[j] * s for j, s in enumerate(streams))


# --------------------------------------------------------------------------- time mixing
def shifted(x, mu, before=None):
    """Each row part of the way to the row ahead of it (zeros, or ``before``, ahead of the first)."""
    first = np.zeros_like(x[:1]) if before is None else before[None]
    return x + (np.concatenate([first, x[:-1]]) - x) * mu


def decays(z, w1, w2, w0):
    """[T, heads * dim], each in (0, 1)."""
    return np.exp(-np.exp(np.tanh(z @ w1.T) @ w2.T + w0))


def wkv_scan(r, k, v, w, u, S=None):
    """One head, token by token: the query reads the state and, through the bonus, the current token; then the state decays
    row by row and takes the token in.  Returns (outputs, final state)."""
    S = np.zeros((k.shape[1], v.shape[1])) if S is None else S.copy()
    out = np.zeros_like(v)
    for t in range(r.shape[0]):
        out[t] = S.T @ r[t] + (r[t] * u * k[t]).sum() * v[t]
        S = w[t][:, None] * S + np.outer(k[t], v[t])
    return out, S


def wkv(x, w, p, m, eps):
    H, d, T = m["heads"], m["dim"], x.shape[0]
    at = {s: shifted(x, w[f"{p}mu.{s}"]) for s in "rkvgw"}
    r, k, v = ((at[s] @ w[p + s].T).reshape(T, H, d) for s in "rkv")
    dec = decays(at["w"], w[p + "w1"], w[p + "w2"], w[p + "w0"]).reshape(T, H, d)
    o = np.stack([wkv_scan(r[:, h], k[:, h], v[:, h], dec[:, h], w[p + "u"][h])[0] for h in range(H)], 1)
    return (unit_rms(o, eps).reshape(T, H * d) * w[p + "norm"] * silu(at["g"] @ w[p + "g"].T)) @ w[p + "o"].T


# --------------------------------------------------------------------------- attention
def bucket(n, rows, far):
    """Row of the bias table for a distance: its own up to half of the table, then in logarithmic steps up to ``far``."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def capped(s, cap):
    return cap * np.tanh(s / cap)


def visible(i, j, size, keep):
    return j <= i and (i - j < size or j < keep)


def mixed_attention(q, k, v, m, rel, talk):
    """q [T, H, d] over k [T, G, d], v [T, G, vd] (consecutive query heads share a key head): capped scores, a bias by
    distance, scores mixed over heads, a window with kept first tokens, a softmax with one more in its denominator."""
    T, H = q.shape[:2]
    per = H // k.shape[1]
    mask = m.get("mask") or {}
    size, keep = mask.get("size") or T, mask.get("keep_first") or 0
    table = np.array([rel[bucket(n, len(rel), m["bias_max"])] for n in range(T)])
    out = np.zeros((T, H, v.shape[2]))
    kh, vh = np.repeat(k, per, axis=1), np.repeat(v, per, axis=1)
    for i in range(T):
        js = np.array([j for j in range(i + 1) if visible(i, j, size, keep)])
        s = np.einsum("hd,jhd->hj", q[i], kh[js]) * m["scale"]
        s = talk @ (capped(s, m["softcap"]) + table[i - js].T)
        top = np.maximum(s.max(-1, keepdims=True), 0.0)
        e = np.exp(s - top)
        out[i] = np.einsum("hj,jhd->hd", e / (np.exp(-top) + e.sum(-1, keepdims=True)), vh[js])
    return out


def attention(x, w, p, m, eps):
    """Queries and keys of unit size; the values are the keys as projected."""
    H, G, d, T = m["heads"], m["kv_heads"], m["dim"], x.shape[0]
    q, k = ((x @ w[p + n].T + w[p + n + ".b"]).reshape(T, -1, d) for n in "qk")
    o = mixed_attention(unit_rms(q, eps), unit_rms(k, eps), k, m, w[p + "rel"], w[p + "talk"])
    return o.reshape(T, H * d) @ w[p + "o"].T


# --------------------------------------------------------------------------- feed-forward
def gated(x, w, p):
    return (silu(x @ w[p + "gate"].T) * (x @ w[p + "up"].T)) @ w[p + "down"].T


def choose(z, top):
    """(expert ids, weights): the scores of the largest as they are."""
    s = softmax(z)
    ids = np.argsort(-s, kind="stable")[:top]
    return ids, s[ids]


def experts(x, w, p, f):
    out = np.zeros_like(x)
    z = x @ w[p + "router"].T
    for t in range(x.shape[0]):
        for e, g in zip(*choose(z[t], f["router"]["top"])):
            out[t] += g * gated(x[t : t + 1], w, f"{p}e{e}.")[0]
    return out


def feed_forward(x, w, p, f):
    return gated(x, w, p) if f["kind"] == "dense" else experts(x, w, p, f)


# --------------------------------------------------------------------------- model
def forward(cfg, w, tokens):
    """(what every layer hands on [layers, T, width], logits [T, vocab])."""
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    results, handed = [x], []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mix = wkv if layer["type"] == "wkv" else attention
        x = x + grouped_norm(mix(x, w, p + "mix.", layer["mixer"], eps), w[p + "norm1"], groups, eps)
        if layer["mlp"] is not None:
            x = x + grouped_norm(feed_forward(x, w, p + "mlp.", layer["mlp"]), w[p + "norm2"], groups, eps)
        results.append(x)
        x = depth_average(results, w[p + "dwa"])
        handed.append(x)
    return np.stack(handed), grouped_norm(x, w["final.norm"], groups, eps) @ w["embed"].T


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[1][-1].argmax()))
    return toks[len(prompt) :]


# --------------------------------------------------------------------------- small random models
def rwkv(heads, dim, rank=5):
    return {"heads": heads, "dim": dim, "_rank": rank}


def attn(heads, kv_heads, dim, size, keep=0, softcap=20.0, rows=8, far=40, scale=0.3):
    """``rows``: of the bias table."""
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "softcap": softcap, "bias_max": far,
            "mask": {"size": size, "keep_first": keep}, "_rows": rows}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(n, top, ff):
    return {"kind": "moe", "router": {"experts": n, "top": top}, "expert": {"ff": ff}}


def config(width, vocab, layers, groups=2, eps=1e-5, embed_scale=3.0):
    """``layers``: (mixer, feed-forward or None)."""
    return {"architecture": "Netovik", "width": width, "vocab": vocab, "norm": {"eps": eps, "groups": groups},
            "embedding": {"scale": embed_scale},
            "layers": [{"type": "attention" if "kv_heads" in m else "wkv", "mixer": m, "mlp": f} for m, f in layers]}


def random_weights(cfg, seed=0, peak=3.0, decay=-2.0):
    """bfloat16-representable weights; ``peak`` scales the head mixing, so that attention is far from uniform; ``decay``: mean
    of the decays' offsets."""
    g = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, out, inp, gain=1.0):
        w[name] = bf16(g.standard_normal((out, inp)) * gain / math.sqrt(inp))

    def vec(name, n, gain=1.0, mean=0.0):
        w[name] = bf16(mean + gain * g.standard_normal(n))

    def triple(p, ff):
        mat(p + "gate", ff, W)
        mat(p + "up", ff, W)
        mat(p + "down", W, ff)

    w["embed"] = bf16(g.standard_normal((V, W)) / math.sqrt(cfg["embedding"]["scale"]))
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        x = p + "mix."
        c = m["heads"] * m["dim"]
        vec(p + "norm1", W, 0.2, 1.0)
        if layer["type"] == "wkv":
            for s in "rkvgw":
                vec(x + "mu." + s, W, 0.3, 0.5)
            for s in "rkvg":
                mat(x + s, c, W)
            mat(x + "w1", m["_rank"], W)
            mat(x + "w2", c, m["_rank"])
            vec(x + "w0", c, 1.5, decay)
            w[x + "u"] = bf16(g.standard_normal((m["heads"], m["dim"])))
            vec(x + "norm", c, 0.2, 1.0)
        else:
            for s, rows in (("q", c), ("k", m["kv_heads"] * m["dim"])):
                mat(x + s, rows, W)
                vec(f"{x}{s}.b", rows, 0.5)
            w[x + "rel"] = bf16(g.standard_normal((m["_rows"], m["heads"])))
            w[x + "talk"] = bf16(g.standard_normal((m["heads"], m["heads"])) * peak / math.sqrt(m["heads"]))
        mat(x + "o", W, c)
        if f is not None:
            vec(p + "norm2", W, 0.2, 1.0)
            if f["kind"] == "dense":
                triple(p + "mlp.", f["ff"])
            else:
                mat(p + "mlp.router", f["router"]["experts"], W, 2.0)
                for e in range(f["router"]["experts"]):
                    triple(f"{p}mlp.e{e}.", f["expert"]["ff"])
        vec(p + "dwa", i + 2, 0.3, 0.5)
    vec("final.norm", W, 0.2, 1.0)
    return w
