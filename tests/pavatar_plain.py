"""Plain, slow float64 statement of the Pavatar design: one function per mechanism, whole sequences, no cache and no batch.

A model is (config dict as it stands in config.json, {tensor name: float64 array}).  Nothing here comes from the package:
the tests compare the engine with these functions."""
import math

import numpy as np

from sokirax_plain import rotate_heads, rotation, silu, softmax, unit_rms  # noqa: F401  (plain statements as well)
from vefilix_plain import bf16, rms_norm, write_model  # noqa: F401


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def softplus(z):
    return np.log1p(np.exp(-np.abs(z))) + np.maximum(z, 0.0)


# --------------------------------------------------------------------------- attention
def causal(q, k, v, scale):
    """Softmax attention of q [T, H, d] over k [T, G, d], v [T, G, vd]; consecutive query heads share a key head."""
    T, H = q.shape[:2]
    per = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        for h in range(H):
            out[i, h] = softmax(k[: i + 1, h // per] @ q[i, h] * scale) @ v[: i + 1, h // per]
    return out


def temperature(pos, coef, every):
    """Factor on a query: grows with the logarithm of how many stretches of ``every`` positions lie behind it."""
    return 1.0 + coef * np.log(np.floor((pos + 1) / every) + 1.0)


def mix_values(v, first, lam):
    return (1.0 - lam) * v + lam * first


def biased_attention(x, w, p, m, first):
    """Unrotated attention with projection biases, values mixed with those of an earlier layer (``first``, None: this layer
    is the earliest), one output gate per head.  Returns (output [T, width], this layer's own values)."""
    H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = x.shape[0]
    q, k, v = (x @ w[p + n].T + w[p + n + ".b"] for n in "qkv")
    q, k, own = q.reshape(T, H, d), k.reshape(T, G, d), v.reshape(T, G, vd)
    if m.get("q_temp"):
        q = q * temperature(np.arange(T), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
    mixed = mix_values(own, first, float(w[p + "vmix"])) if m.get("v_mix") and first is not None else own
    o = causal(q, k, mixed, m["scale"]) * sigmoid(x @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * vd) @ w[p + "o"].T, own


def rotated_attention(x, w, p, m, eps):
    """Attention with a norm per query / key head, partial rotation and a gate on every output value."""
    H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = x.shape[0]
    q, k, v = (x @ w[p + "q"].T).reshape(T, H, d), (x @ w[p + "k"].T).reshape(T, G, d), (x @ w[p + "v"].T).reshape(T, G, vd)
    q, k = rms_norm(q, w[p + "q.norm"], eps), rms_norm(k, w[p + "k.norm"], eps)
    o = causal(rotate_heads(q, m["rot"]), rotate_heads(k, m["rot"]), v, m["scale"]).reshape(T, H * vd)
    return (o * sigmoid(x @ w[p + "g"].T)) @ w[p + "o"].T


# --------------------------------------------------------------------------- gated delta rule
def short_conv(u, taps):
    """Depthwise causal convolution over time of u [T, channels] with taps [channels, n], the last on the current row."""
    n = taps.shape[1]
    pad = np.concatenate([np.zeros((n - 1, u.shape[1])), u])
    return sum(pad[j : j + u.shape[0]] * taps[:, j] for j in range(n))


def unit(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def delta_scan(q, k, v, decay, beta, S=None):
    """One head, token by token: the state decays (row by row: decay [T, dim] or [T, 1]), the part of v that the key already
    recalls is taken off, the rest is written, the query reads.  Returns (outputs [T, vdim], final state)."""
    S = np.zeros((k.shape[1], v.shape[1])) if S is None else S.copy()
    out = np.zeros((q.shape[0], v.shape[1]))
    for t in range(q.shape[0]):
        S = decay[t][:, None] * S
        S = S + np.outer(k[t], beta[t] * (v[t] - S.T @ k[t]))
        out[t] = S.T @ q[t]
    return out, S


def log_decay(x, w, p, m, per_channel):
    """[T, heads, dim] or [T, heads, 1]: never positive."""
    H, T = m["heads"], x.shape[0]
    z = (x @ w[p + "a1"].T) @ w[p + "a2"].T if per_channel else x @ w[p + "a"].T
    return -np.exp(w[p + "A_log"])[None, :, None] * softplus(z + w[p + "dt_bias"]).reshape(T, H, -1)


def delta(x, w, p, m, eps, per_channel):
    """``per_channel``: a decay per key channel and a sigmoid output gate, both of low rank; else a decay per head and a
    silu gate."""
    H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = x.shape[0]
    q, k, v = (silu(short_conv(x @ w[p + n].T, w[f"{p}{n}.conv"])) for n in "qkv")
    q, k, v = unit(q.reshape(T, G, d)) * d ** -0.5, unit(k.reshape(T, G, d)), v.reshape(T, H, vd)
    beta, g = sigmoid(x @ w[p + "b"].T), np.exp(log_decay(x, w, p, m, per_channel))
    o = np.stack([delta_scan(q[:, h // (H // G)], k[:, h // (H // G)], v[:, h], g[:, h], beta[:, h])[0] for h in range(H)], 1)
    gate = sigmoid((x @ w[p + "g1"].T) @ w[p + "g2"].T) if per_channel else silu(x @ w[p + "g"].T)
    return ((unit_rms(o, eps) * w[p + "norm"]).reshape(T, H * vd) * gate) @ w[p + "o"].T


# --------------------------------------------------------------------------- layers
def mixer(x, w, p, layer, eps, first):
    """(output [T, width], the values later layers mix in)"""
    m = layer["mixer"]
    if layer["type"] == "attention":
        y, own = biased_attention(x, w, p, m, first)
        return y, own if m.get("v_mix") and first is None else first
    if layer["type"] == "delta":
        return delta(x, w, p, m, eps, False), first
    left, right = rotated_attention(x, w, p + "left.", m["left"], eps), delta(x, w, p + "right.", m["right"], eps, True)
    return 0.5 * (rms_norm(left, w[p + "left.out"], eps) + rms_norm(right, w[p + "right.out"], eps)), first


def choose(z, correction, top, scale):
    """(expert ids, weights): the correction takes part in the choice only."""
    s = softmax(z)
    ids = np.argsort(-(s + correction), kind="stable")[:top]
    return ids, s[ids] / (s[ids].sum() + 1e-20) * scale


def expert(x, w, p):
    return np.maximum(x @ w[p + "up"].T, 0.0) ** 2 @ w[p + "down"].T


def experts(x, w, p, f):
    out = np.zeros_like(x)
    z = x @ w[p + "router"].T
    for t in range(x.shape[0]):
        for e, g in zip(*choose(z[t], w[p + "correction"], f["router"]["top"], f["router"]["scale"])):
            out[t] += g * expert(x[t : t + 1], w, f"{p}e{e}.")[0]
    return out


def forward(cfg, w, tokens):
    """(residual stream after every layer [layers, T, width], logits [T, vocab])."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    streams, first = [], None
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms_norm(x, w[p + "norm1"], eps)
        y, first = mixer(h, w, p + "mix.", layer, eps, first)
        x = x + y + (experts(h, w, p + "mlp.", layer["mlp"]) if layer["mlp"] is not None else 0.0)
        streams.append(x)
    cap = cfg["logit_softcap"]
    return np.stack(streams), cap * np.tanh(rms_norm(x, w["final.norm"], eps) @ w["embed"].T / cap)


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[1][-1].argmax()))
    return toks[len(prompt) :]


# --------------------------------------------------------------------------- small random models
def attn(heads, kv_heads, dim, vdim, q_temp=None, v_mix=True, scale=0.2):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if q_temp is not None:
        m["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    return m


def rotated(heads, kv_heads, dim, vdim, rot, scale=0.2):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot, "scale": scale}


def dlt(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def parallel(left, right):
    return {"left": left, "right": right}


def moe(n, top, ff, scale=1.0):
    return {"kind": "moe", "router": {"experts": n, "top": top, "scale": scale}, "expert": {"ff": ff}}


def config(width, vocab, layers, eps=1e-5, embed_scale=3.0, softcap=20.0):
    """``layers``: (mixer, feed-forward or None)."""
    kind = lambda m: "parallel" if "left" in m else "delta" if "conv" in m else "attention"
    return {"architecture": "Pavatar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed_scale},
            "logit_softcap": softcap, "layers": [{"type": kind(m), "mixer": m, "mlp": f} for m, f in layers]}


def random_weights(cfg, seed=0, peak=2.0, rank=None):
    """bfloat16-representable weights; ``peak`` scales the queries, so that attention is far from uniform; ``rank``: of the
    low-rank decay and gate projections."""
    g = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, out, inp, gain=1.0):
        w[name] = bf16(g.standard_normal((out, inp)) * gain / math.sqrt(inp))

    def vec(name, n, gain=1.0, mean=0.0):
        w[name] = bf16(mean + gain * g.standard_normal(n))

    def qkv(p, m, q_gain=1.0):
        mat(p + "q", m["heads"] * m["dim"], W, q_gain)
        mat(p + "k", m["kv_heads"] * m["dim"], W)
        mat(p + "v", m["kv_heads"] * m["vdim"], W)
        mat(p + "o", W, m["heads"] * m["vdim"], 1.5)

    def delta_rule(p, m, per_channel):
        H, G, d, vd, n = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        r = rank or max(1, d // 3)
        for name, rows in (("q", G * d), ("k", G * d), ("v", H * vd)):
            mat(p + name, rows, W)
            w[f"{p}{name}.conv"] = bf16(g.standard_normal((rows, n)) / math.sqrt(n))
        mat(p + "b", H, W)
        vec(p + "A_log", H, 1.0, -1.0)
        vec(p + "norm", vd, 0.2, 1.0)
        vec(p + "dt_bias", H * d if per_channel else H, 1.0, -1.5)
        if per_channel:
            for a in "ag":
                mat(f"{p}{a}1", r, W)
                mat(f"{p}{a}2", H * (d if a == "a" else vd), r)
        else:
            mat(p + "a", H, W)
            mat(p + "g", H * vd, W)
        mat(p + "o", W, H * vd, 1.5)

    w["embed"] = bf16(g.standard_normal((V, W)))
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        vec(p + "norm1", W, 0.2, 1.0)
        if layer["type"] == "attention":
            qkv(p + "mix.", m, peak)
            for n, rows in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                vec(f"{p}mix.{n}.b", rows, 0.5)
            w[p + "mix.vmix"] = bf16(np.float64(0.2 + 0.6 * g.random()))
            mat(p + "mix.g", m["heads"], W)
        elif layer["type"] == "delta":
            delta_rule(p + "mix.", m, False)
        else:
            l = m["left"]
            qkv(p + "mix.left.", l)
            vec(p + "mix.left.q.norm", l["dim"], 0.2, peak)
            vec(p + "mix.left.k.norm", l["dim"], 0.2, 1.0)
            mat(p + "mix.left.g", l["heads"] * l["vdim"], W)
            delta_rule(p + "mix.right.", m["right"], True)
            for side in ("left", "right"):
                vec(f"{p}mix.{side}.out", W, 0.2, 1.0)
        if f is not None:
            for e in range(f["router"]["experts"]):
                mat(f"{p}mlp.e{e}.up", f["expert"]["ff"], W)
                mat(f"{p}mlp.e{e}.down", W, f["expert"]["ff"])
            mat(p + "mlp.router", f["router"]["experts"], W, 2.0)
            vec(p + "mlp.correction", f["router"]["experts"], 0.1)
    vec("final.norm", W, 0.2, 1.0)
    return w
