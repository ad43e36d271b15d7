"""Models that describe every layer on its own: configuration readers and the weight loader.

``READERS`` maps the lower-case ``"architecture"`` of a ``config.json`` to the function that turns it into a
:class:`ModelConfig` with ``layer_specs``.

Vefilix: layer norm (weight and bias) after each sum, ``x <- norm(alpha x + branch(x))``, with latent attention in a
sliding window (a softmax sink per head, YaRN-scaled rotation, later layers reading an earlier layer's cached rows) and
ungated squared-relu feed-forward blocks; the embedding and the output pass norms of their own."""
from __future__ import annotations

import math
from typing import Any, Callable, Dict, List, Optional, Tuple

import numpy as np
import torch

from ..formats.layered import LayeredCheckpoint
from .config import (FeedForwardSpec, LatentAttentionSpec, LayerSpec, ModelConfig, RopeScaling, RotarySpec,
                     UnsupportedArchitecture)
from .weights import LayerWeights, LinearWeight, MLAWeights, ModelWeights, QTensor, StreamedLayers, shard_range


# --------------------------------------------------------------------------- configuration
def _yarn(s: Optional[Dict[str, Any]], dims: int) -> Optional[RopeScaling]:
    if not s:
        return None
    factor = float(s["factor"])
    # the ramp may end past the last pair (dims - 1), and cos / sin carry the magnitude whatever the factor
    return RopeScaling("yarn", factor, float(s["original"]), float(s["fast"]), float(s["slow"]), ramp_limit=dims - 1,
                       magnitude=0.1 * math.log(factor) + 1.0)


def _latent_mixer(m: Dict[str, Any], layer: int) -> LatentAttentionSpec:
    rot = m["rot"]
    dims = int(rot["dims"])
    if dims != int(m["rot_dim"]):
        raise UnsupportedArchitecture(f"layer {layer}: the rotation covers {dims} of {m['rot_dim']} positional dimensions")
    mask = m.get("mask") or {}
    src = m.get("kv_from")
    return LatentAttentionSpec(heads=int(m["heads"]), nope_dim=int(m["dim"]), rope_dim=int(m["rot_dim"]), v_dim=int(m["vdim"]),
                               kv_rank=int(m["kv_rank"]), scale=float(m["scale"]),
                               rotary=RotarySpec(dims, float(rot["base"]), _yarn(rot.get("scaling"), dims)),
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


def layered_config(arch: str, vocab: int, width: int, specs: List[LayerSpec], eps: float, norm_kind: str,
                   residual_alpha: float, embed_norm: bool, name: str = "") -> ModelConfig:
    m0 = specs[0].mixer
    ffn = max([l.ffn.size for l in specs if l.ffn is not None], default=0)
    return ModelConfig(arch=arch, name=name, vocab_size=vocab, hidden_size=width, n_layers=len(specs), n_heads=m0.heads,
                       n_kv_heads=1, head_dim=max(l.mixer.row_dim for l in specs), ffn_size=ffn, rms_eps=eps,
                       rope_theta=m0.rotary.base, rope_dim=m0.rotary.dims, attn_scale=m0.scale, context_length=1 << 20,
                       layer_specs=specs, norm_kind=norm_kind, residual_alpha=residual_alpha, embed_norm=embed_norm)


READERS: Dict[str, Callable[[LayeredCheckpoint], ModelConfig]] = {"vefilix": _vefilix_config}


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
    if 0 < resident_layers < n:
        layers = StreamedLayers(lambda i: _load_layer(src, cfg.layer_specs[i], i, tp_rank, tp_size), n, resident_layers)
    else:
        layers = [_load_layer(src, cfg.layer_specs[i], i, tp_rank, tp_size) for i in range(n)]
    v0, v1 = shard_range(cfg.vocab_size, tp_rank, tp_size) if cfg.vocab_size % tp_size == 0 else (0, cfg.vocab_size)
    mw = ModelWeights(cfg, src.matrix("embed"), layers, src.vector("final.norm"), LinearWeight([src.matrix("head", rows=(v0, v1))]),
                      [], tp_rank, tp_size, 0, 1, 0, v0)
    mw.out_norm_bias = src.vector("final.norm.b")
    mw.embed_norm, mw.embed_norm_bias = src.vector("embed.norm"), src.vector("embed.norm.b")
    return mw
