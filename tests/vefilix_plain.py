"""Plain, slow float64 statement of the Vefilix design: one function per mechanism, whole sequences, no cache and no batch.

A model is (config dict as it stands in config.json, {tensor name: float64 array}).  Nothing here comes from the package:
the tests compare the engine with these functions."""
import json
import math
import os
import struct

import numpy as np


# --------------------------------------------------------------------------- mechanisms
def layer_norm(x, weight, bias, eps):
    mean = x.mean(-1, keepdims=True)
    dev = x - mean
    return dev / np.sqrt((dev * dev).mean(-1, keepdims=True) + eps) * weight + bias


def rms_norm(x, weight, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * weight


def frequencies(rot):
    """(angle per position of each pair, factor on cos and sin)."""
    d, base, s = rot["dims"], float(rot["base"]), rot.get("scaling")
    f = [base ** (-2.0 * i / d) for i in range(d // 2)]
    if not s:
        return np.array(f), 1.0

    def dim(turns):
        return d * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(dim(s["fast"])), 0)
    hi = min(math.ceil(dim(s["slow"])), d - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * r + fi * (1 - r))
    return np.array(out), 0.1 * math.log(s["factor"]) + 1.0


def rotate(v, pos, rot):
    """Rotation of the first rot.dims values of v at position pos; value i is paired with value i + dims / 2."""
    f, mag = frequencies(rot)
    half = rot["dims"] // 2
    out = v.copy()
    for i in range(half):
        c, s = math.cos(pos * f[i]) * mag, math.sin(pos * f[i]) * mag
        out[i] = v[i] * c - v[i + half] * s
        out[i + half] = v[i + half] * c + v[i] * s
    return out


def softmax_with_sink(scores, sink):
    top = max(float(scores.max()), sink)
    e = np.exp(scores - top)
    return e / (e.sum() + math.exp(sink - top))


def visible(i, window):
    """Positions that position i sees."""
    return range(max(0, i - window + 1), i + 1)


def cached_rows(x, w, p, m, eps):
    """(latent, rotated key part) of every position."""
    y = x @ w[p + "dkv"].T
    lat = rms_norm(y[:, : m["kv_rank"]], w[p + "dkv.norm"], eps)
    keys = np.stack([rotate(y[t, m["kv_rank"] :], t, m["rot"]) for t in range(x.shape[0])])
    return lat, keys


def latent_attention(x, w, p, m, rows):
    H, d, r, vd = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    lat, kr = rows
    T = x.shape[0]
    q = (x @ w[p + "q"].T).reshape(T, H, d + r)
    kn = (lat @ w[p + "uk"].T).reshape(T, H, d)
    v = (lat @ w[p + "uv"].T).reshape(T, H, vd)
    out = np.zeros((T, H, vd))
    for i in range(T):
        seen = list(visible(i, m["mask"]["size"]))
        for h in range(H):
            qr = rotate(q[i, h, d:], i, m["rot"])
            s = (kn[seen, h] @ q[i, h, :d] + kr[seen] @ qr) * m["scale"]
            out[i, h] = softmax_with_sink(s, float(w[p + "sink"][h])) @ v[seen, h]
    return out.reshape(T, H * vd) @ w[p + "o"].T


def feed_forward(x, w, p):
    return np.square(np.maximum(x @ w[p + "up"].T, 0.0)) @ w[p + "down"].T


def forward(cfg, w, tokens):
    """(residual stream after every layer [layers, T, width], logits [T, vocab])."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = layer_norm(w["embed"][np.asarray(tokens)], w["embed.norm"], w["embed.norm.b"], eps)
    rows, streams = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        src = m.get("kv_from")
        if src is None:
            src = i
            rows[i] = cached_rows(x, w, p + "mix.", m, eps)
        x = layer_norm(alpha * x + latent_attention(x, w, p + "mix.", m, rows[src]), w[p + "norm1"], w[p + "norm1.b"], eps)
        if layer["mlp"] is not None:
            x = layer_norm(alpha * x + feed_forward(x, w, p + "mlp."), w[p + "norm2"], w[p + "norm2.b"], eps)
        streams.append(x)
    return np.stack(streams), layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[1][-1].argmax()))
    return toks[len(prompt) :]


# --------------------------------------------------------------------------- small random models
def mixer(heads, dim, rot_dim, vdim, rank, window, scale=0.2, base=10000.0, scaling=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "mask": {"size": window}, "scale": scale,
         "rot": {"base": base, "dims": rot_dim, "scaling": scaling}}
    if scaling is None:
        del m["rot"]["scaling"]
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def config(width, vocab, layers, alpha=2.0, eps=1e-5):
    """``layers``: (mixer, feed-forward size or None)."""
    return {"architecture": "Vefilix", "width": width, "vocab": vocab, "postln_alpha": alpha, "norm": {"eps": eps},
            "layers": [{"type": "latent_attention", "mixer": m, "mlp": None if f is None else {"kind": "dense", "ff": f}}
                       for m, f in layers]}


def bf16(x):
    """Round to bfloat16 (to nearest even), returned as float64."""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    u = ((u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)).astype(np.uint32)
    return u.view(np.float32).astype(np.float64)


def random_weights(cfg, seed=0, peak=2.0):
    """bfloat16-representable weights; ``peak`` scales the queries, so that attention is far from uniform."""
    g = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, out, inp, gain=1.0):
        w[name] = bf16(g.standard_normal((out, inp)) * gain / math.sqrt(inp))

    def norm(name, n, bias=True):
        w[name] = bf16(1 + 0.2 * g.standard_normal(n))
        if bias:
            w[name + ".b"] = bf16(0.2 * g.standard_normal(n))

    mat("embed", V, W, math.sqrt(W))
    norm("embed.norm", W)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, r = m["heads"], m["kv_rank"]
        mat(p + "mix.q", H * (m["dim"] + m["rot_dim"]), W, peak)
        if m.get("kv_from") is None:
            mat(p + "mix.dkv", r + m["rot_dim"], W)
            norm(p + "mix.dkv.norm", r, bias=False)
        mat(p + "mix.uk", H * m["dim"], r)
        mat(p + "mix.uv", H * m["vdim"], r)
        w[p + "mix.sink"] = bf16(1 + g.standard_normal(H))
        mat(p + "mix.o", W, H * m["vdim"], 1.5)
        norm(p + "norm1", W)
        if layer["mlp"] is not None:
            mat(p + "mlp.up", layer["mlp"]["ff"], W)
            mat(p + "mlp.down", W, layer["mlp"]["ff"])
            norm(p + "norm2", W)
    norm("final.norm", W)
    mat("head", V, W)
    return w


def write_model(path, cfg, w):
    """config.json and model.safetensors (bfloat16) in directory ``path``."""
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, off = {}, [], 0
    for name, x in w.items():
        raw = (np.ascontiguousarray(x, dtype=np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        head[name] = {"dtype": "BF16", "shape": list(x.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    h = json.dumps(head).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))
    return str(path)
