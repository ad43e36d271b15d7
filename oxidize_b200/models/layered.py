"""Models that describe every layer on its own: configuration readers and the weight loader.

``READERS`` maps the lower-case ``"architecture"`` of a ``config.json`` to the function that turns it into a
:class:`ModelConfig` with ``layer_specs``.

Vefilix: layer norm (weight and bias) after each sum, ``x <- norm(alpha x + branch(x))``, with latent attention in a
sliding window (a softmax sink per head, YaRN-scaled rotation, later layers reading an earlier layer's cached rows) and
ungated squared-relu feed-forward blocks; the embedding and the output pass norms of their own.

Sokirax: RMS norms on both sides of every branch, x <- x + norm_b(branch(norm_a(x))); grouped-query attention in a window
(per-head q / k norm, partial YaRN rotation), or such attention (norm over the whole projection, a softmax sink per head)
beside retention on the same input; gated feed-forward blocks, dense or routed experts with a shared one; a layer may use an
earlier layer's weights.

Pavatar: one RMS norm that mixer and feed-forward block both read, x <- x + mixer(h) + ffn(h); unrotated attention (biases,
a query factor that grows with the position, values mixed with an earlier layer's, a gate per head), the gated delta rule with
a decay per head, or rotated attention (q / k norms, a gate per output value) beside the gated delta rule with a decay per key
channel, each side with a norm of its own; routed squared-relu experts with a correction of the choice; a scaled embedding that
is the output head as well, and soft-capped logits.

Netovik: RMS norms in groups on the branches' outputs only, x <- x + norm(branch(x)), and after every layer a learned weighted
sum of the embedding and all results so far; RWKV time mixing, or unrotated attention whose values are its keys (soft-capped
scores, a bias by distance, scores mixed over the heads, a window with kept first tokens, one in the softmax denominator);
gated feed-forward blocks, dense or routed with the scores as they are; a scaled embedding that is the output head as well."""
from __future__ import annotations

import dataclasses
import functools
import math
from typing import Any, Callable, Dict, List, Optional, Tuple

import numpy as np
import torch

from ..formats.layered import LayeredCheckpoint
from .config import (AttentionSpec, DeltaSpec, FeedForwardSpec, LatentAttentionSpec, LayerSpec, ModelConfig, MoESpec,
                     ParallelSpec, RetentionSpec, RopeScaling, RotarySpec, UnsupportedArchitecture, WkvSpec, distance_bucket, pad_to)
from .weights import (DeltaWeights, ExpertWeights, LayerWeights, LinearWeight, MLAWeights, ModelWeights, QTensor,
                      StreamedLayers, WkvWeights, shard_range)


# --------------------------------------------------------------------------- configuration
def _yarn(s: Optional[Dict[str, Any]], dims: int) -> Optional[RopeScaling]:
    if not s:
        return None
    factor = float(s["factor"])
    # the ramp may end past the last pair (dims - 1), and cos / sin carry the magnitude whatever the factor
    return RopeScaling("yarn", factor, float(s["original"]), float(s["fast"]), float(s["slow"]), ramp_limit=dims - 1,
                       magnitude=0.1 * math.log(factor) + 1.0)


def _rotary(rot: Dict[str, Any]) -> RotarySpec:
    dims = int(rot["dims"])
    return RotarySpec(dims, float(rot["base"]), _yarn(rot.get("scaling"), dims))


def _latent_mixer(m: Dict[str, Any], layer: int) -> LatentAttentionSpec:
    rot = m["rot"]
    dims = int(rot["dims"])
    if dims != int(m["rot_dim"]):
        raise UnsupportedArchitecture(f"layer {layer}: the rotation covers {dims} of {m['rot_dim']} positional dimensions")
    mask = m.get("mask") or {}
    src = m.get("kv_from")
    return LatentAttentionSpec(heads=int(m["heads"]), nope_dim=int(m["dim"]), rope_dim=int(m["rot_dim"]), v_dim=int(m["vdim"]),
                               kv_rank=int(m["kv_rank"]), scale=float(m["scale"]),
                               rotary=_rotary(rot),
                               window=int(mask.get("size") or 0), sink=True, kv_from=None if src is None else int(src))


def _dense_ffn(f: Optional[Dict[str, Any]], layer: int) -> Optional[FeedForwardSpec]:
    if f is None:
        return None
    if f.get("kind") != "dense":
        raise UnsupportedArchitecture(f"layer {layer}: feed-forward kind {f.get('kind')!r}")
    return FeedForwardSpec(int(f["ff"]), "relu2")


def check_sources(specs: List[LayerSpec]) -> None:
    """A layer that reads another layer's cached rows needs an earlier layer that writes rows of the same geometry."""
    for i, l in enumerate(specs):
        j = l.mixer.kv_from
        if j is None:
            continue
        if not 0 <= j < i or specs[j].mixer.kv_from is not None:
            raise ValueError(f"layer {i}: kv_from {j} is not an earlier layer with cache rows of its own")
        a, b = l.mixer, specs[j].mixer
        if (a.kv_rank, a.rope_dim, a.rotary) != (b.kv_rank, b.rope_dim, b.rotary):
            raise ValueError(f"layer {i} and its kv_from layer {j} differ in latent size or rotation")


def _vefilix_config(ck: LayeredCheckpoint) -> ModelConfig:
    c = ck.config
    specs = []
    for i, l in enumerate(c["layers"]):
        if l.get("type") != "latent_attention":
            raise UnsupportedArchitecture(f"layer {i}: mixer type {l.get('type')!r}")
        specs.append(LayerSpec(_latent_mixer(l["mixer"], i), _dense_ffn(l.get("mlp"), i)))
    check_sources(specs)
    return layered_config("vefilix", int(c["vocab"]), int(c["width"]), specs, eps=float(c["norm"]["eps"]), norm_kind="layer",
                          residual_alpha=float(c["postln_alpha"]), embed_norm=True, name=str(ck.get("general.name", "")))


def _attention(m: Dict[str, Any], qk_norm: str, sink: bool, layer: int, **kw) -> AttentionSpec:
    mask = m.get("mask") or {}
    a = AttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), v_dim=int(m["vdim"]),
                      scale=float(m["scale"]), rotary=_rotary(m["rot"]) if m.get("rot") else None,
                      window=int(mask.get("size") or 0), sink=sink, qk_norm=qk_norm, **kw)
    if a.heads % a.kv_heads:
        raise UnsupportedArchitecture(f"layer {layer}: {a.heads} query heads over {a.kv_heads} key / value heads")
    if a.rotary is not None and (a.rotary.dims % 2 or a.rotary.dims > a.dim):
        raise UnsupportedArchitecture(f"layer {layer}: rotation of {a.rotary.dims} of {a.dim} values per head")
    return a


def _retention(m: Dict[str, Any], layer: int) -> RetentionSpec:
    r = RetentionSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), [float(d) for d in m["decay"]], _rotary(m["rot"]))
    if len(r.decay) != r.heads:
        raise ValueError(f"layer {layer}: {len(r.decay)} decays for {r.heads} heads")
    if any(not 0.0 < d <= 1.0 for d in r.decay):
        raise UnsupportedArchitecture(f"layer {layer}: decays must lie in (0, 1]")
    if r.rotary.dims % 2 or r.rotary.dims > r.dim:
        raise UnsupportedArchitecture(f"layer {layer}: rotation of {r.rotary.dims} of {r.dim} values per head")
    return r


def _gated_ffn(f: Optional[Dict[str, Any]], layer: int):
    if f is None:
        return None
    if f.get("kind") == "dense":
        return FeedForwardSpec(int(f["ff"]), "silu", gated=True)
    if f.get("kind") != "moe":
        raise UnsupportedArchitecture(f"layer {layer}: feed-forward kind {f.get('kind')!r}")
    shared = f.get("shared")
    m = MoESpec(int(f["router"]["experts"]), int(f["router"]["top"]), FeedForwardSpec(int(f["expert"]["ff"]), "silu", True),
                FeedForwardSpec(int(shared["ff"]), "silu", True) if shared else None)
    if not 1 <= m.n_experts_used <= m.n_experts:
        raise ValueError(f"layer {layer}: {m.n_experts_used} of {m.n_experts} experts per token")
    return m


def check_shared_weights(specs: List[LayerSpec]) -> None:
    """A layer that uses another layer's weights names one that has weights of its own and the same geometry."""
    for i, l in enumerate(specs):
        j = l.weights_of
        if j is None:
            continue
        if not 0 <= j < len(specs) or specs[j].weights_of is not None:
            raise ValueError(f"layer {i}: weights_of {j} is not a layer with weights of its own")
        if (l.mixer, l.ffn) != (specs[j].mixer, specs[j].ffn):
            raise ValueError(f"layer {i} uses the weights of layer {j} but differs from it")


def _sokirax_config(ck: LayeredCheckpoint) -> ModelConfig:
    c = ck.config
    specs = []
    for i, l in enumerate(c["layers"]):
        m = l["mixer"]
        if l.get("type") == "attention":
            mixer = _attention(m, "head", False, i)
        elif l.get("type") == "parallel":
            mixer = ParallelSpec(_attention(m["left"], "full", True, i), _retention(m["right"], i), float(m["left_scale"]),
                                 float(m["right_scale"]))
        else:
            raise UnsupportedArchitecture(f"layer {i}: mixer type {l.get('type')!r}")
        src = l.get("weights_of")
        specs.append(LayerSpec(mixer, _gated_ffn(l.get("mlp"), i), None if src is None else int(src)))
    check_shared_weights(specs)
    return layered_config("sokirax", int(c["vocab"]), int(c["width"]), specs, eps=float(c["norm"]["eps"]), norm_kind="rms",
                          norm_placement="sandwich", name=str(ck.get("general.name", "")))


def _unrotated(m: Dict[str, Any], layer: int) -> AttentionSpec:
    t = m.get("q_temp") or {}
    a = _attention(dict(m, rot=None), "", False, layer, bias=True, temp_coef=float(t.get("coef", 0.0)),
                   temp_every=float(t.get("every", 1.0)), v_mix=bool(m.get("v_mix")), gate="head")
    if not a.temp_every > 0:
        raise ValueError(f"layer {layer}: query temperature every {a.temp_every} positions")
    return a


def _delta(ck: LayeredCheckpoint, m: Dict[str, Any], prefix: str, layer: int, low_rank: bool) -> DeltaSpec:
    rank = (lambda n: int(ck.tensors[f"{prefix}{n}"].shape[0])) if low_rank else (lambda n: 0)
    d = DeltaSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]), rank("a1"), rank("g1"))
    if d.heads % d.kv_heads:
        raise UnsupportedArchitecture(f"layer {layer}: {d.heads} value heads over {d.kv_heads} query / key heads")
    if d.conv < 1:
        raise ValueError(f"layer {layer}: a convolution over {d.conv} tokens")
    return d


def _corrected_experts(f: Optional[Dict[str, Any]], layer: int) -> Optional[MoESpec]:
    if f is None:
        return None
    if f.get("kind") != "moe":
        raise UnsupportedArchitecture(f"layer {layer}: feed-forward kind {f.get('kind')!r}")
    r = f["router"]
    m = MoESpec(int(r["experts"]), int(r["top"]), FeedForwardSpec(int(f["expert"]["ff"]), "relu2"),
                expert_weights_scale=float(r.get("scale", 1.0)), correction=True)
    if not 1 <= m.n_experts_used <= m.n_experts:
        raise ValueError(f"layer {layer}: {m.n_experts_used} of {m.n_experts} experts per token")
    return m


def check_value_mixing(specs: List[LayerSpec]) -> None:
    """Layers that mix their values with the first such layer's have values of its geometry."""
    mixed = [(i, l.attention) for i, l in enumerate(specs) if isinstance(l.attention, AttentionSpec) and l.attention.v_mix]
    for i, a in mixed:
        f = mixed[0][1]
        if (a.kv_heads, a.v_dim) != (f.kv_heads, f.v_dim):
            raise ValueError(f"layer {i} mixes values of {a.kv_heads} x {a.v_dim} with layer {mixed[0][0]}'s of "
                             f"{f.kv_heads} x {f.v_dim}")


def _pavatar_config(ck: LayeredCheckpoint) -> ModelConfig:
    c = ck.config
    specs = []
    for i, l in enumerate(c["layers"]):
        m, p = l["mixer"], f"l{i}.mix."
        if l.get("type") == "attention":
            mixer = _unrotated(m, i)
        elif l.get("type") == "delta":
            mixer = _delta(ck, m, p, i, False)
        elif l.get("type") == "parallel":
            mixer = ParallelSpec(_attention(m["left"], "head", False, i, gate="value"), _delta(ck, m["right"], p + "right.", i, True),
                                 0.5, 0.5, norms=True)
        else:
            raise UnsupportedArchitecture(f"layer {i}: mixer type {l.get('type')!r}")
        specs.append(LayerSpec(mixer, _corrected_experts(l.get("mlp"), i)))
    check_value_mixing(specs)
    cfg = layered_config("pavatar", int(c["vocab"]), int(c["width"]), specs, eps=float(c["norm"]["eps"]), norm_kind="rms",
                         norm_placement="parallel", name=str(ck.get("general.name", "")))
    cfg.embedding_scale = float((c.get("embedding") or {}).get("scale") or 1.0)
    cfg.final_softcap = float(c.get("logit_softcap") or 0.0)
    cfg.tie_embeddings = True
    return cfg


def _joint_attention(ck: LayeredCheckpoint, m: Dict[str, Any], prefix: str, layer: int) -> AttentionSpec:
    """Unrotated attention whose heads' scores are mixed and whose values are the keys as projected."""
    rows = int(ck.tensors[prefix + "rel"].shape[0])
    a = _attention(dict(m, rot=None), "unit", False, layer, bias=True, keep_first=int((m.get("mask") or {}).get("keep_first") or 0),
                   softcap=float(m.get("softcap") or 0.0), bias_rows=rows, bias_max=int(m["bias_max"]), talk=True, unit_sink=True,
                   shared_kv=True)
    if a.v_dim != a.dim:
        raise UnsupportedArchitecture(f"layer {layer}: values of {a.v_dim} that are keys of {a.dim}")
    if rows < 2 or rows % 2 or a.bias_max <= rows // 2:
        raise UnsupportedArchitecture(f"layer {layer}: {rows} biases for distances up to {a.bias_max}")
    return a


def _wkv(ck: LayeredCheckpoint, m: Dict[str, Any], prefix: str, hidden: int) -> WkvSpec:
    return WkvSpec(int(m["heads"]), int(m["dim"]), int(ck.tensors[prefix + "w1"].shape[0]), hidden)


def _unnormed_experts(f: Optional[Dict[str, Any]], layer: int):
    """Gated blocks; routed experts are weighed by their scores as they are."""
    s = _gated_ffn(f, layer)
    return dataclasses.replace(s, expert_weights_norm=False) if isinstance(s, MoESpec) else s


def _netovik_config(ck: LayeredCheckpoint) -> ModelConfig:
    c = ck.config
    width, specs = int(c["width"]), []
    for i, l in enumerate(c["layers"]):
        p = f"l{i}.mix."
        if l.get("type") == "attention":
            mixer = _joint_attention(ck, l["mixer"], p, i)
        elif l.get("type") == "wkv":
            mixer = _wkv(ck, l["mixer"], p, width)
        else:
            raise UnsupportedArchitecture(f"layer {i}: mixer type {l.get('type')!r}")
        specs.append(LayerSpec(mixer, _unnormed_experts(l.get("mlp"), i)))
    cfg = layered_config("netovik", int(c["vocab"]), width, specs, eps=float(c["norm"]["eps"]), norm_kind="rms",
                         norm_placement="output", name=str(ck.get("general.name", "")))
    cfg.norm_groups = int(c["norm"].get("groups") or 1)
    if cfg.norm_groups < 1 or width % cfg.norm_groups:
        raise UnsupportedArchitecture(f"a norm over {cfg.norm_groups} parts of {width} values")
    cfg.depth_average = True
    cfg.embedding_scale = float((c.get("embedding") or {}).get("scale", 1.0))
    cfg.tie_embeddings = True
    return cfg


def layered_config(arch: str, vocab: int, width: int, specs: List[LayerSpec], eps: float, norm_kind: str,
                   residual_alpha: float = 1.0, embed_norm: bool = False, name: str = "",
                   norm_placement: str = "after_sum") -> ModelConfig:
    atts = [l.attention for l in specs if l.attention is not None]
    m0 = atts[0] if atts else specs[0].recurrent
    rot = next((p.rotary for l in specs for p in (l.attention, l.recurrent) if p is not None and p.rotary is not None), None)
    ffn = max([l.ffn.size for l in specs if l.ffn is not None], default=0)
    return ModelConfig(arch=arch, name=name, vocab_size=vocab, hidden_size=width, n_layers=len(specs), n_heads=m0.heads,
                       n_kv_heads=max([a.kv_heads for a in atts], default=1),
                       head_dim=max([a.cache_shape[2] for a in atts], default=16), ffn_size=ffn, rms_eps=eps,
                       rope_theta=rot.base if rot else 10000.0, rope_dim=rot.dims if rot else 0, attn_scale=getattr(m0, "scale", 0.0),
                       context_length=1 << 20, layer_specs=specs, norm_kind=norm_kind, residual_alpha=residual_alpha,
                       embed_norm=embed_norm, norm_placement=norm_placement)


READERS: Dict[str, Callable[[LayeredCheckpoint], ModelConfig]] = {"vefilix": _vefilix_config, "sokirax": _sokirax_config,
                                                                      "pavatar": _pavatar_config, "netovik": _netovik_config}


def config_from_layered(ck: LayeredCheckpoint) -> ModelConfig:
    if ck.architecture not in READERS:
        raise UnsupportedArchitecture(f"unknown architecture {ck.architecture!r}; layer-list checkpoints: {sorted(READERS)}")
    return READERS[ck.architecture](ck)


# --------------------------------------------------------------------------- weights
class LayeredWeightSource:
    """Reads (slices of) tensors of a layer-list checkpoint into device tensors of the compute type."""

    def __init__(self, ck: LayeredCheckpoint, device, act_dtype: torch.dtype):
        self.ck, self.device, self.act_dtype = ck, torch.device(device), act_dtype

    def tensor(self, name: str) -> torch.Tensor:
        a, dt = self.ck.raw(name)
        if dt == "BF16":
            return torch.from_numpy(np.array(a).view(np.int16)).view(torch.bfloat16)
        return torch.from_numpy(np.array(a))

    def vector(self, name: str) -> torch.Tensor:
        return self.tensor(name).float().reshape(-1).to(self.device)

    def dense(self, name: str, rows: Tuple[int, int] = None, cols: Tuple[int, int] = None) -> torch.Tensor:
        t = self.tensor(name)
        if rows is not None:
            t = t[rows[0] : rows[1]]
        if cols is not None:
            t = t[:, cols[0] : cols[1]]
        return t.to(self.act_dtype).contiguous().to(self.device)

    def matrix(self, name: str, rows: Tuple[int, int] = None, cols: Tuple[int, int] = None) -> QTensor:
        return dense_qtensor(self.dense(name, rows, cols))


def dense_qtensor(w: torch.Tensor) -> QTensor:
    return QTensor("F32" if w.dtype == torch.float32 else "BF16", w, (w.shape[0], w.shape[1]))


def latent_weights(spec: LatentAttentionSpec, q: torch.Tensor, dkv: Optional[torch.Tensor], dkv_norm: Optional[torch.Tensor],
                   uk: torch.Tensor, uv: torch.Tensor, sink: Optional[torch.Tensor]) -> MLAWeights:
    """Mixer weights in the layout the forward pass uses: the query and down projections share one matrix (one product
    over the layer's input), the up-projections stand per head."""
    H = q.shape[0] // spec.qk_dim
    rows = q if dkv is None else torch.cat([q, dkv], dim=0)
    return MLAWeights(kv_a=None, kv_a_norm=dkv_norm, w_uk=uk.reshape(H, spec.nope_dim, spec.kv_rank).contiguous(),
                      w_uv=uv.reshape(H, spec.v_dim, spec.kv_rank).contiguous(),
                      q=LinearWeight([dense_qtensor(rows.contiguous())]), sink=sink)


def pad_heads(t: torch.Tensor, heads: int, width: int, dim: int = 0) -> torch.Tensor:
    """Every head's values along axis ``dim`` followed by zeros up to ``width`` of them."""
    n = t.shape[dim] // heads
    if n == width:
        return t
    shape = list(t.shape)
    parts = t.reshape(shape[:dim] + [heads, n] + shape[dim + 1 :])
    pad = torch.zeros(shape[:dim] + [heads, width - n] + shape[dim + 1 :], dtype=t.dtype, device=t.device)
    return torch.cat([parts, pad], dim=dim + 1).reshape(shape[:dim] + [heads * width] + shape[dim + 1 :])


def pad_rows(t: torch.Tensor, rows: int) -> torch.Tensor:
    """``t`` followed by zero rows up to ``rows``."""
    return t if t.shape[0] == rows else torch.cat([t, t.new_zeros(rows - t.shape[0], *t.shape[1:])])


def pad_cols(t: torch.Tensor, cols: int) -> torch.Tensor:
    return torch.nn.functional.pad(t, (0, cols - t.shape[1])).contiguous()


def delta_weights(d: DeltaSpec, t: Dict[str, torch.Tensor], act_dtype: torch.dtype) -> Tuple[List[torch.Tensor], DeltaWeights]:
    """Delta-rule tensors (as stored) in the layout the forward pass uses: (rows over the layer's input q | k | v | gate |
    decay | beta, what acts behind them)."""
    K, V, H, G = d.k_width, d.v_width, d.heads, d.kv_heads
    ins = [pad_heads(t["q"], G, K), pad_heads(t["k"], G, K), pad_heads(t["v"], H, V)]
    taps = torch.cat([pad_heads(t["q.conv"].float(), G, K), pad_heads(t["k.conv"].float(), G, K), pad_heads(t["v.conv"].float(), H, V)])
    w = DeltaWeights(conv=taps.t().contiguous(), a_log=t["A_log"].float().contiguous(),
                     norm=torch.nn.functional.pad(t["norm"].float(), (0, V - d.v_dim)).contiguous(), dt_bias=t["dt_bias"].float().contiguous())
    if d.gate_rank:
        ins.append(pad_rows(t["g1"], d.gate_dim))
        w.gate_up = pad_cols(pad_heads(t["g2"], H, V), d.gate_dim).to(act_dtype)
    else:
        ins.append(pad_heads(t["g"], H, V))
    if d.decay_rank:
        ins.append(pad_rows(t["a1"], d.decay_dim))
        w.decay_up = pad_cols(pad_heads(t["a2"], H, K), d.decay_dim).to(act_dtype)
        w.dt_bias = pad_heads(w.dt_bias, H, K).contiguous()
    else:
        ins.append(pad_rows(t["a"], d.decay_dim))
    ins.append(pad_rows(t["b"], pad_to(H, 8)))
    return ins, w


@functools.lru_cache(None)
def distance_rows(rows: int, far: int) -> Tuple[int, ...]:
    """Bias rows of the distances 0, 1, ... up to the first that has the last row (as have all beyond it)."""
    out = [0]
    while out[-1] < rows - 1:
        out.append(distance_bucket(len(out), rows, far))
    return tuple(out)


def distance_bias(rel: torch.Tensor, far: int, mix: Optional[torch.Tensor]) -> torch.Tensor:
    """Bias table [rows, heads] to [heads, distances], what every head's mixed score gets from it."""
    t = rel.double()[torch.tensor(distance_rows(rel.shape[0], far), device=rel.device)].t()
    return (t if mix is None else mix.double() @ t).float().contiguous()


def wkv_weights(k: WkvSpec, t: Dict[str, torch.Tensor], act_dtype: torch.dtype) -> Dict[str, Any]:
    """Time-mixing tensors (as stored) in the layout the forward pass uses."""
    H, W = k.heads, k.k_width
    pad, ld = lambda n: pad_heads(t[n].float().reshape(-1), H, W).contiguous(), pad_to(k.hidden, 8)
    w = WkvWeights(mu=torch.stack([t["mu." + n].float().reshape(-1) for n in "rkvgw"]).contiguous(),
                   proj=torch.stack([pad_cols(pad_heads(t[n], H, W), ld) for n in "rkvg"]).contiguous(),
                   decay_down=LinearWeight([dense_qtensor(pad_cols(pad_rows(t["w1"], k.decay_dim), ld))]),
                   decay_up=pad_cols(pad_heads(t["w2"], H, W), k.decay_dim).to(act_dtype), decay_base=pad("w0"), bonus=pad("u"),
                   norm=pad("norm"))
    return {"wqkv": None, "wo": LinearWeight([dense_qtensor(pad_heads(t["o"], H, W, dim=1).contiguous())]), "wkv": w}


def listed_mixer(spec: LayerSpec, att: Dict[str, torch.Tensor], rec: Dict[str, torch.Tensor]) -> Dict[str, Any]:
    """Attention and / or recurrent tensors (as stored) of one layer in the layout the forward pass uses: one matrix over
    the layer's input, attention q | k | v | gate then retention q | k | v | gate or the delta rule's rows, and one output
    matrix over both mixers' heads (two where each side's output has a norm of its own), every head padded with zeros to its
    kernel width."""
    ins, outs, kw = [], [], {}
    a, r, d = spec.attention, spec.retention, spec.delta
    ret, bias = rec, None
    if a is not None:
        parts = (("q", a.heads), ("k", a.kv_heads)) + (() if a.shared_kv else (("v", a.kv_heads),))
        for n, heads in parts:
            ins.append(pad_heads(att[n], heads, a.width))
        if a.gate:
            ins.append(pad_rows(att["g"], a.gate_dim) if a.gate == "head" else pad_heads(att["g"], a.heads, a.width))
        if a.bias:
            bias = torch.cat([pad_heads(att[n + ".b"].float(), heads, a.width) for n, heads in parts])
        kw["v_mix"] = att["vmix"].float().reshape(1).contiguous() if a.v_mix else None
        outs.append(pad_heads(att["o"], a.heads, a.width, dim=1))
        if a.qk_norm in ("head", "full"):
            full = a.qk_norm == "full"
            kw["q_norm"] = pad_heads(att["q.norm"], a.heads if full else 1, a.width).contiguous()
            kw["k_norm"] = pad_heads(att["k.norm"], a.kv_heads if full else 1, a.width).contiguous()
        kw["sink"] = att["sink"] if a.sink else None
        if a.unit_sink:
            kw["sink"] = torch.zeros(a.heads, dtype=torch.float32, device=att["q"].device)
        if a.talk:
            kw["score_mix"] = att["talk"].float().reshape(a.heads, a.heads).contiguous()
        if a.bias_rows:
            kw["score_bias"] = distance_bias(att["rel"], a.bias_max, kw.get("score_mix"))
    if r is not None:
        for n, width in (("q", r.k_width), ("k", r.k_width), ("v", r.v_width), ("g", r.v_width)):
            ins.append(pad_heads(ret[n], r.heads, width))
        outs.append(pad_heads(ret["o"], r.heads, r.v_width, dim=1))
    if d is not None:
        rows, kw["delta"] = delta_weights(d, rec, rec["q"].dtype)
        ins += rows
        outs.append(pad_heads(rec["o"], d.heads, d.v_width, dim=1))
    w_in = torch.cat(ins, dim=0).contiguous()
    kw["wqkv"] = LinearWeight([dense_qtensor(w_in)], None if bias is None else pad_rows(bias, w_in.shape[0]).contiguous())
    if isinstance(spec.mixer, ParallelSpec) and spec.mixer.norms:
        kw["wo"], kw["wo_right"] = (LinearWeight([dense_qtensor(o.contiguous())]) for o in outs)
    else:
        kw["wo"] = LinearWeight([dense_qtensor(torch.cat(outs, dim=1).contiguous())])
    return kw


def gated_pair(gate: Optional[torch.Tensor], up: torch.Tensor, down: torch.Tensor, size: int, rows: int = 0,
               cols: int = 0) -> Tuple[QTensor, QTensor]:
    """([gate | up], down), or (up, down) without a gate, with ``size`` feed-forward columns, the input padded to ``cols``
    values and the output to ``rows``."""
    def grow(t, n, k):
        return torch.nn.functional.pad(t, (0, max(k - t.shape[1], 0), 0, max(n - t.shape[0], 0)))

    gu = torch.cat([grow(t, size, cols) for t in (gate, up) if t is not None], dim=0).contiguous()
    return dense_qtensor(gu), dense_qtensor(grow(down, rows, size).contiguous())


def listed_experts(spec: MoESpec, triples, hidden: int) -> ExpertWeights:
    """The experts' (gate or None, up, down), stacked; inner sizes are multiples of the grouped product's k-block."""
    h64 = pad_to(hidden, 64)
    pairs = [gated_pair(g, u, d, pad_to(spec.expert.size, 64), h64, h64) for g, u, d in triples]
    ex = ExpertWeights([p[0] for p in pairs], [p[1] for p in pairs])
    for name in ("gate_up", "down"):
        lst = getattr(ex, name)
        n, k = lst[0].shape
        stack = dense_qtensor(torch.cat([q.data for q in lst], dim=0).contiguous())
        setattr(ex, name + "_stack", stack)
        for i, q in enumerate(lst):
            q.data = stack.data[i * n : (i + 1) * n]
    return ex


def _load_listed(src: LayeredWeightSource, cfg: ModelConfig, i: int) -> LayerWeights:
    """A layer with norms on both sides of its branches."""
    spec, p = cfg.layer_specs[i], f"l{i}"

    def mixer(prefix: str, names, part) -> Dict[str, torch.Tensor]:
        return {n: src.dense(f"{p}.mix.{prefix}{n}") for n in names} if part is not None else {}

    both = isinstance(spec.mixer, ParallelSpec)
    a, r = spec.attention, spec.retention
    att, ret = mixer("left." if both else "", ("q", "k", "v", "o"), a), mixer("right." if both else "", ("q", "k", "v", "g", "o"), r)
    for n in (("q.norm", "k.norm") if a is not None and a.qk_norm else ()) + (("sink",) if a is not None and a.sink else ()):
        att[n] = src.vector(f"{p}.mix.{'left.' if both else ''}{n}")
    lw = LayerWeights(attn_norm=src.vector(f"{p}.norm1"), post_attn_norm=src.vector(f"{p}.norm1b"), ffn_norm=None,
                      **listed_mixer(spec, att, ret))
    f = spec.ffn
    if f is None:
        return lw
    lw.ffn_norm, lw.post_ffn_norm = src.vector(f"{p}.norm2"), src.vector(f"{p}.norm2b")

    def triple(prefix: str):
        return tuple(src.dense(f"{p}.mlp.{prefix}{n}") for n in ("gate", "up", "down"))

    gated_block(lw, f, cfg.hidden_size, triple)
    if isinstance(f, MoESpec):
        lw.router = src.matrix(f"{p}.mlp.router")
        if f.shared is not None:
            gu, down = gated_pair(*triple("shared."), f.shared.pad_size)
            lw.shared_gate_up, lw.shared_down = LinearWeight([gu]), LinearWeight([down])
    return lw


def _load_joint(src: LayeredWeightSource, cfg: ModelConfig, i: int) -> LayerWeights:
    """A layer with one norm that both branches read."""
    spec, p = cfg.layer_specs[i], f"l{i}"
    a, d, f = spec.attention, spec.delta, spec.ffn
    both = isinstance(spec.mixer, ParallelSpec)

    def mixer(prefix: str, matrices, vectors) -> Dict[str, torch.Tensor]:
        out = {n: src.dense(f"{p}.mix.{prefix}{n}") for n in matrices}
        out.update({n: src.vector(f"{p}.mix.{prefix}{n}") for n in vectors})
        return out

    att, rec = {}, {}
    if a is not None:
        att = mixer("left." if both else "", ["q", "k", "v", "o"] + (["g"] if a.gate else []),
                    (["q.b", "k.b", "v.b"] if a.bias else []) + (["q.norm", "k.norm"] if a.qk_norm else [])
                    + (["vmix"] if a.v_mix else []))
    if d is not None:
        rec = mixer("right." if both else "", ["q", "k", "v", "o", "b", "q.conv", "k.conv", "v.conv"]
                    + (["a1", "a2"] if d.decay_rank else ["a"]) + (["g1", "g2"] if d.gate_rank else ["g"]), ["A_log", "dt_bias", "norm"])
    lw = LayerWeights(attn_norm=src.vector(f"{p}.norm1"), ffn_norm=None, **listed_mixer(spec, att, rec))
    if both:
        lw.out_norms = (src.vector(f"{p}.mix.left.out"), src.vector(f"{p}.mix.right.out"))
    if f is not None:
        lw.router, lw.router_bias = src.matrix(f"{p}.mlp.router"), src.vector(f"{p}.mlp.correction")
        lw.experts = listed_experts(f, [(None, src.dense(f"{p}.mlp.e{e}.up"), src.dense(f"{p}.mlp.e{e}.down"))
                                        for e in range(f.n_experts)], cfg.hidden_size)
    return lw


def gated_block(lw: LayerWeights, f, hidden: int, triple) -> None:
    """Feed-forward weights of a layer, dense or routed; ``triple(prefix)``: (gate, up, down) as stored."""
    if isinstance(f, MoESpec):
        lw.experts = listed_experts(f, (triple(f"e{e}.") for e in range(f.n_experts)), hidden)
    else:
        gu, down = gated_pair(*triple(""), f.pad_size)
        lw.w_gate_up, lw.w_down = LinearWeight([gu]), LinearWeight([down])


def _load_output_normed(src: LayeredWeightSource, cfg: ModelConfig, i: int) -> LayerWeights:
    """A layer with norms on its branches' outputs only."""
    spec, p = cfg.layer_specs[i], f"l{i}"
    dense, vectors = lambda *names: {n: src.dense(f"{p}.mix.{n}") for n in names}, lambda *names: {n: src.vector(f"{p}.mix.{n}") for n in names}
    a = spec.attention
    if spec.wkv is not None:
        kw = wkv_weights(spec.wkv, {**dense("r", "k", "v", "g", "w1", "w2", "o"), **vectors(*("mu." + n for n in "rkvgw"), "w0", "u", "norm")},
                         src.act_dtype)
    else:
        att = {**dense("q", "k", "o"), **vectors("q.b", "k.b", "talk"), "rel": src.vector(f"{p}.mix.rel").reshape(a.bias_rows, a.heads)}
        kw = listed_mixer(spec, att, {})
    lw = LayerWeights(attn_norm=None, post_attn_norm=src.vector(f"{p}.norm1"), ffn_norm=None, **kw)
    lw.depth = src.vector(f"{p}.dwa") if cfg.depth_average else None
    if spec.ffn is not None:
        lw.post_ffn_norm = src.vector(f"{p}.norm2")
        if isinstance(spec.ffn, MoESpec):
            lw.router = src.matrix(f"{p}.mlp.router")
        gated_block(lw, spec.ffn, cfg.hidden_size, lambda prefix: tuple(src.dense(f"{p}.mlp.{prefix}{n}") for n in ("gate", "up", "down")))
    return lw


def _load_layer(src: LayeredWeightSource, spec: LayerSpec, i: int, tp_rank: int, tp_size: int) -> LayerWeights:
    p, m = f"l{i}", spec.mixer
    h0, h1 = shard_range(m.heads, tp_rank, tp_size)
    own = m.kv_from is None
    mla = latent_weights(m, src.dense(f"{p}.mix.q", rows=(h0 * m.qk_dim, h1 * m.qk_dim)),
                         src.dense(f"{p}.mix.dkv") if own else None, src.vector(f"{p}.mix.dkv.norm") if own else None,
                         src.dense(f"{p}.mix.uk", rows=(h0 * m.nope_dim, h1 * m.nope_dim)),
                         src.dense(f"{p}.mix.uv", rows=(h0 * m.v_dim, h1 * m.v_dim)),
                         src.vector(f"{p}.mix.sink")[h0:h1].contiguous() if m.sink else None)
    lw = LayerWeights(attn_norm=src.vector(f"{p}.norm1"), attn_norm_bias=src.vector(f"{p}.norm1.b"), wqkv=None,
                      wo=LinearWeight([src.matrix(f"{p}.mix.o", cols=(h0 * m.v_dim, h1 * m.v_dim))]), ffn_norm=None, mla=mla)
    if spec.ffn is not None:
        f0, f1 = shard_range(spec.ffn.size, tp_rank, tp_size)
        lw.ffn_norm, lw.ffn_norm_bias = src.vector(f"{p}.norm2"), src.vector(f"{p}.norm2.b")
        lw.w_up = LinearWeight([src.matrix(f"{p}.mlp.up", rows=(f0, f1))])
        lw.w_down = LinearWeight([src.matrix(f"{p}.mlp.down", cols=(f0, f1))])
    return lw


def load_layered_weights(ck: LayeredCheckpoint, cfg: ModelConfig, device="cpu", act_dtype: torch.dtype = torch.float32,
                         tp_rank: int = 0, tp_size: int = 1, resident_layers: int = 0) -> ModelWeights:
    """This rank's shard of a layer-list checkpoint: heads and feed-forward columns are cut, the latent projection is
    replicated (every rank caches the whole latent row)."""
    src = LayeredWeightSource(ck, device, act_dtype)
    n = cfg.n_layers
    whole = {"sandwich": _load_listed, "parallel": _load_joint, "output": _load_output_normed}.get(cfg.norm_placement)
    if whole is not None and tp_size > 1:
        raise ValueError("a norm over all heads and per-sequence states are not sharded: run this model with tp_size = 1")

    def load(i: int) -> LayerWeights:
        return whole(src, cfg, i) if whole is not None else _load_layer(src, cfg.layer_specs[i], i, tp_rank, tp_size)

    source = [i if l.weights_of is None else l.weights_of for i, l in enumerate(cfg.layer_specs)]
    if 0 < resident_layers < n:
        layers = StreamedLayers(lambda i: load(source[i]), n, resident_layers)
    else:
        own = {i: load(i) for i in sorted(set(source))}
        layers = [own[i] for i in source]
    v0, v1 = shard_range(cfg.vocab_size, tp_rank, tp_size) if cfg.vocab_size % tp_size == 0 else (0, cfg.vocab_size)
    embed = src.matrix("embed")
    head = embed if cfg.tie_embeddings else src.matrix("head", rows=(v0, v1))
    mw = ModelWeights(cfg, embed, layers, src.vector("final.norm"), LinearWeight([head]), [], tp_rank, tp_size, 0, 1, 0, v0)
    if cfg.norm_kind == "layer":
        mw.out_norm_bias = src.vector("final.norm.b")
    if cfg.embed_norm:
        mw.embed_norm, mw.embed_norm_bias = src.vector("embed.norm"), src.vector("embed.norm.b")
    return mw
