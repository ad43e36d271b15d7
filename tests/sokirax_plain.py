"""Plain, slow float64 statement of the Sokirax design: one function per mechanism, whole sequences, no cache and no batch.

A model is (config dict as it stands in config.json, {tensor name: float64 array}).  Nothing here comes from the package:
the tests compare the engine with these functions."""
import math

import numpy as np

from vefilix_plain import bf16, frequencies, rms_norm, visible, write_model  # noqa: F401  (plain statements as well)


# --------------------------------------------------------------------------- mechanisms
def rotate_heads(x, rot):
    """x [T, heads, dim]: value i of the first rot.dims values of every head is paired with value i + dims / 2."""
    f, mag = frequencies(rot)
    half = rot["dims"] // 2
    a = np.arange(x.shape[0])[:, None] * f[None, :]
    c, s = (np.cos(a) * mag)[:, None, :], (np.sin(a) * mag)[:, None, :]
    out = x.copy()
    u, v = x[..., :half], x[..., half : 2 * half]
    out[..., :half] = u * c - v * s
    out[..., half : 2 * half] = v * c + u * s
    return out


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def silu(z):
    return z / (1.0 + np.exp(-z))


def softmax(scores, sink=None):
    """``sink``: a logit that joins the denominator only."""
    top = scores.max() if sink is None else max(scores.max(), sink)
    e = np.exp(scores - top)
    return e / (e.sum() + (0.0 if sink is None else math.exp(sink - top)))


def attention(x, w, p, m, eps, full_norm, sink):
    """Grouped-query attention in a window, up to its output projection: [T, heads * vdim].  ``full_norm``: one norm over
    all heads of q (and of k) instead of one per head."""
    H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = x.shape[0]
    q, k, v = x @ w[p + "q"].T, x @ w[p + "k"].T, x @ w[p + "v"].T
    if full_norm:
        q, k = rms_norm(q, w[p + "q.norm"], eps), rms_norm(k, w[p + "k.norm"], eps)
    q, k, v = q.reshape(T, H, d), k.reshape(T, G, d), v.reshape(T, G, vd)
    if not full_norm:
        q, k = rms_norm(q, w[p + "q.norm"], eps), rms_norm(k, w[p + "k.norm"], eps)
    q, k = rotate_heads(q, m["rot"]), rotate_heads(k, m["rot"])
    out = np.zeros((T, H, vd))
    for i in range(T):
        seen = list(visible(i, m["mask"]["size"]))
        for h in range(H):
            g = h // (H // G)
            out[i, h] = softmax(k[seen, g] @ q[i, h] * m["scale"], float(w[p + "sink"][h]) if sink else None) @ v[seen, g]
    return out.reshape(T, H * vd)


def retention_scan(q, k, v, decay):
    """S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t for one head, token by token."""
    S = np.zeros((k.shape[1], v.shape[1]))
    out = np.zeros((q.shape[0], v.shape[1]))
    for t in range(q.shape[0]):
        S = decay * S + np.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out


def retention(x, w, p, m, eps):
    """Linear attention with a fixed decay per head, up to its output projection: [T, heads * vdim]."""
    H, d, vd = m["heads"], m["dim"], m["vdim"]
    T = x.shape[0]
    q = rotate_heads((x @ w[p + "q"].T).reshape(T, H, d), m["rot"])
    k = rotate_heads((x @ w[p + "k"].T).reshape(T, H, d), m["rot"]) * d ** -0.5
    v = (x @ w[p + "v"].T).reshape(T, H, vd)
    o = np.stack([retention_scan(q[:, h], k[:, h], v[:, h], m["decay"][h]) for h in range(H)], axis=1)
    return unit_rms(o, eps).reshape(T, H * vd) * silu(x @ w[p + "g"].T)


def mixer(x, w, p, layer, eps):
    m = layer["mixer"]
    if layer["type"] == "attention":
        return attention(x, w, p, m, eps, full_norm=False, sink=False) @ w[p + "o"].T
    left = attention(x, w, p + "left.", m["left"], eps, full_norm=True, sink=True) @ w[p + "left.o"].T
    right = retention(x, w, p + "right.", m["right"], eps) @ w[p + "right.o"].T
    return m["left_scale"] * left + m["right_scale"] * right


def gated_ffn(x, w, p):
    return (silu(x @ w[p + "gate"].T) * (x @ w[p + "up"].T)) @ w[p + "down"].T


def choose(logits, top):
    """(expert ids, weights): the largest logits and the softmax over those alone."""
    ids = np.argsort(-logits, kind="stable")[:top]
    return ids, softmax(logits[ids])


def feed_forward(x, w, p, f):
    if f["kind"] == "dense":
        return gated_ffn(x, w, p)
    out = np.zeros_like(x)
    z = x @ w[p + "router"].T
    for t in range(x.shape[0]):
        for e, g in zip(*choose(z[t], f["router"]["top"])):
            out[t] += g * gated_ffn(x[t : t + 1], w, f"{p}e{e}.")[0]
    return out + gated_ffn(x, w, p + "shared.") if f.get("shared") else out


def forward(cfg, w, tokens):
    """(residual stream after every layer [layers, T, width], logits [T, vocab])."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{layer.get('weights_of', i)}."
        x = x + rms_norm(mixer(rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", layer, eps), w[p + "norm1b"], eps)
        if layer["mlp"] is not None:
            y = feed_forward(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"])
            x = x + rms_norm(y, w[p + "norm2b"], eps)
        streams.append(x)
    return np.stack(streams), rms_norm(x, w["final.norm"], eps) @ w["head"].T


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[1][-1].argmax()))
    return toks[len(prompt) :]


# --------------------------------------------------------------------------- small random models
def rotation(dims, base=10000.0, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling is not None:
        r["scaling"] = scaling
    return r


def attn(heads, kv_heads, dim, vdim, window, rot, scale=0.2):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "rot": rot, "scale": scale}


def ret(heads, dim, vdim, decay, rot):
    assert len(decay) == heads
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay), "rot": rot}


def parallel(left, right, left_scale, right_scale):
    return {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    f = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared is not None:
        f["shared"] = {"ff": shared}
    return f


def config(width, vocab, layers, eps=1e-5):
    """``layers``: (mixer, feed-forward or None), or the number of the layer whose weights a layer uses."""
    out = []
    for l in layers:
        if isinstance(l, int):
            out.append(dict(out[l], weights_of=l))
        else:
            out.append({"type": "parallel" if "left" in l[0] else "attention", "mixer": l[0], "mlp": l[1]})
    return {"architecture": "Sokirax", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": out}


def random_weights(cfg, seed=0, peak=2.0):
    """bfloat16-representable weights; ``peak`` scales the query norms, so that attention is far from uniform."""
    g = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, out, inp, gain=1.0):
        w[name] = bf16(g.standard_normal((out, inp)) * gain / math.sqrt(inp))

    def norm(name, n, gain=1.0):
        w[name] = bf16(gain * (1 + 0.2 * g.standard_normal(n)))

    def ffn(p, ff):
        mat(p + "gate", ff, W)
        mat(p + "up", ff, W)
        mat(p + "down", W, ff)

    def qkv(p, m, nq, nk):
        mat(p + "q", m["heads"] * m["dim"], W)
        mat(p + "k", m["kv_heads"] * m["dim"], W)
        mat(p + "v", m["kv_heads"] * m["vdim"], W)
        norm(p + "q.norm", nq, peak)
        norm(p + "k.norm", nk)
        mat(p + "o", W, m["heads"] * m["vdim"], 1.5)

    mat("embed", V, W, math.sqrt(W))
    for i, layer in enumerate(cfg["layers"]):
        if "weights_of" in layer:
            continue
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        norm(p + "norm1", W)
        norm(p + "norm1b", W)
        if layer["type"] == "attention":
            qkv(p + "mix.", m, m["dim"], m["dim"])
        else:
            l, r = m["left"], m["right"]
            qkv(p + "mix.left.", l, l["heads"] * l["dim"], l["kv_heads"] * l["dim"])
            w[p + "mix.left.sink"] = bf16(1 + g.standard_normal(l["heads"]))
            for n in ("q", "k"):
                mat(f"{p}mix.right.{n}", r["heads"] * r["dim"], W)
            for n in ("v", "g"):
                mat(f"{p}mix.right.{n}", r["heads"] * r["vdim"], W)
            mat(p + "mix.right.o", W, r["heads"] * r["vdim"], 1.5)
        if f is not None:
            norm(p + "norm2", W)
            norm(p + "norm2b", W)
            if f["kind"] == "dense":
                ffn(p + "mlp.", f["ff"])
            else:
                for e in range(f["router"]["experts"]):
                    ffn(f"{p}mlp.e{e}.", f["expert"]["ff"])
                mat(p + "mlp.router", f["router"]["experts"], W, 2.0)
                if f.get("shared"):
                    ffn(p + "mlp.shared.", f["shared"]["ff"])
    norm("final.norm", W)
    mat("head", V, W)
    return w
