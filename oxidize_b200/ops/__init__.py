"""Operator front door.

CPU tensors run the plain-PyTorch statements in :mod:`oxidize_b200.ops.ref` (the oracle and
the no-GPU execution path).  CUDA tensors always run the hand-written sm_100a kernels in
:mod:`oxidize_b200.ops.cuda`; there is no silent fallback — if the native library is missing
on a GPU machine the call raises.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from . import ref
from ..utils.profiler import instrument


def _cuda():
    from . import cuda as _c

    return _c


def _cuda_latent():
    from . import cuda_latent as _c

    return _c


def _cuda_listed():
    from . import cuda_listed as _c

    return _c


def _cuda_joint():
    from . import cuda_joint as _c

    return _c


def _cuda_wkv():
    from . import cuda_wkv as _c

    return _c


class DepthStreams:
    """The embedding and the layers' results of a step, kept for the weighted sums that go on from layer to layer."""

    def __init__(self, x: torch.Tensor, layers: int):
        self.first = x  # [T, hidden] float32
        self.results = torch.empty(layers, *x.shape, dtype=torch.float32, device=x.device)
        self.n = 0


@dataclass
class NormedPair:
    """Projected outputs of two mixers that pass RMS norms of their own: left_scale * norm(left) + right_scale * norm(right)."""

    left: torch.Tensor
    right: torch.Tensor
    left_norm: torch.Tensor
    right_norm: torch.Tensor
    left_scale: float
    right_scale: float


@dataclass
class RoutedRows:
    """Routed experts ahead of their weighted sum: token t's is sum_j weights[t, j] * rows[index[t, j]]."""

    rows: torch.Tensor  # [T * k, hidden or more]
    index: torch.Tensor  # [T, k] int32
    weights: torch.Tensor  # [T, k] float32


@instrument("linear")
def linear(x: torch.Tensor, w, bias: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """y = x @ W^T (+bias) for a :class:`LinearWeight` (row segments concatenated) or a QTensor."""
    parts = getattr(w, "parts", None)
    if parts is None:
        parts = [w]
    else:
        bias = w.bias if bias is None else bias
    if x.is_cuda:
        if x.dtype == torch.float32 and all(p.qtype == "F32" for p in parts):
            return _cuda_latent().linear_f32(x, parts, bias, out)
        return _cuda().linear(x, parts, bias, out)
    ys = [ref.linear(x, p) for p in parts]
    y = ys[0] if len(ys) == 1 else torch.cat(ys, dim=-1)
    if bias is not None:
        y = (y.float() + bias.float()).to(y.dtype)
    return y


@instrument("embed")
def embed(tokens: torch.Tensor, table, dtype: torch.dtype, scale: float = 1.0) -> torch.Tensor:
    if tokens.is_cuda:
        return _cuda().embed(tokens, table, dtype, scale)
    return ref.embed(tokens, table, scale).to(dtype)


@instrument("rmsnorm")
def rmsnorm(x, w, eps):
    if x.is_cuda:
        return _cuda().add_rmsnorm(x, None, w, eps)[0]
    return ref.rmsnorm(x, w, eps)


@instrument("add_rmsnorm")
def add_rmsnorm(x, residual, w, eps):
    if x.is_cuda:
        return _cuda().add_rmsnorm(x, residual, w, eps)
    return ref.add_rmsnorm(x, residual, w, eps)


@instrument("silu_mul")
def silu_mul(gate_up):
    if gate_up.is_cuda:
        return _cuda().silu_mul(gate_up)
    return ref.silu_mul(gate_up)


@instrument("gelu_mul")
def gelu_mul(gate_up):
    """tanh-GELU(gate) * up on the halves of a fused [T, 2F] projection (GeGLU)."""
    if gate_up.is_cuda:
        return _cuda().gelu_mul(gate_up)
    return ref.gelu_mul(gate_up)


@instrument("branch_norm")
def branch_norm(res, y, w_post, w_next, eps, act_dtype=torch.float32):
    """Norms on both sides of a branch: x = res + rmsnorm(y) * w_post (float32; ``y`` None: x = res) and the next branch's
    input rmsnorm(x) * w_next in ``act_dtype`` (None without ``w_next``)."""
    if res.is_cuda:
        return _cuda_listed().branch_norm(res, y, w_post, w_next, eps, act_dtype)
    return ref.branch_norm(res, y, w_post, w_next, eps, act_dtype)


@instrument("joint_norm")
def joint_norm(res, mix, ffn, w_next, eps, act_dtype=torch.float32):
    """Both branches of a layer join the stream: x = res + mix + ffn (float32) and the next layer's input rmsnorm(x) * w_next
    in ``act_dtype`` (None without ``w_next``).  ``mix``: None, a tensor or a ``NormedPair``; ``ffn``: None, a tensor or
    ``RoutedRows``."""
    if res.is_cuda:
        return _cuda_listed().joint_norm(res, mix, ffn, w_next, eps, act_dtype)
    return ref.joint_norm(res, mix, ffn, w_next, eps, act_dtype)


@instrument("add_normed")
def add_normed(res, y, w, groups, eps, act_dtype=None, streams: Optional[DepthStreams] = None, depth=None):
    """A branch's output joins the stream through a norm in groups: x = res + norm(y) * w in float32, every one of ``groups``
    consecutive parts over its own root mean square; ``y``: a tensor or ``RoutedRows``.  With ``streams`` and ``depth`` [n + 2] x
    becomes the n-th result and what comes back is depth[0] * first + sum_j depth[j + 1] * results[j].  (that, the same in
    ``act_dtype`` or None without one)."""
    if res.is_cuda:
        return _cuda_listed().add_normed(res, y, w, groups, eps, act_dtype, streams, depth)
    return ref.add_normed(res, y, w, groups, eps, act_dtype, streams, depth)


@instrument("grouped_norm")
def grouped_norm(x, w, groups, eps, act_dtype=torch.float32):
    """norm(x) * w, every one of ``groups`` consecutive parts over its own root mean square."""
    if x.is_cuda:
        return _cuda_listed().grouped_norm(x, w, groups, eps, act_dtype)
    return ref.grouped_norm(x, w, groups, eps).to(act_dtype)


@instrument("wkv_mixer")
def wkv_mixer(x, w, spec, meta, state, window, eps, act_dtype=torch.float32):
    """RWKV time mixing of one layer on its float32 input, up to (not including) the output projection: [T, spec.out_dim] in
    ``act_dtype``; ``state`` [slots, heads, k_width, v_width] and ``window`` [slots, 1, hidden] are updated."""
    if x.is_cuda:
        return _cuda_wkv().wkv_mixer(x, w, spec, meta, state, window, eps, act_dtype)
    mixes = ref.token_shift(x, w.mu, meta, window).to(act_dtype)
    mixes = torch.nn.functional.pad(mixes, (0, w.proj.shape[2] - spec.hidden))
    rkvg = torch.stack([(mixes[i].float() @ w.proj[i].float().t()).to(act_dtype) for i in range(4)])
    low = linear(mixes[4], w.decay_down)
    return ref.wkv(rkvg, ref.wkv_log_decay(low, w), w, spec, meta, state, eps).to(act_dtype)


def first_values(z, a, lw, carry):
    """(values of the model's first value-mixing layer [T, kv_heads, width], this layer's share of them) for a layer that mixes
    them into its own; (None, None) elsewhere.  The first such layer leaves its own in ``carry``."""
    if not a.v_mix:
        return None, None
    v = z[:, (a.heads + a.kv_heads) * a.width : a.qkv_dim].unflatten(1, (a.kv_heads, a.width))
    if carry is None:
        raise ValueError("a layer that mixes values needs the step's earlier layers")
    first = carry.setdefault("values", v)
    return (None, None) if first is v else (first, lw.v_mix)


@instrument("listed_mixer")
def listed_mixer(x, lw, spec, ropes, meta, kv, kv_layer, state_layer, eps, carry=None):
    """Attention and / or a recurrence of one listed layer on its normed input, up to (not including) the output projection:
    [T, spec.out_dim], attention heads first, or the two sides apart where each has an output projection of its own.
    ``ropes``: rotations of the two; in a layer with one projection over both, each side's output carries its scale.
    ``carry``: what this step's earlier layers left for later ones."""
    if x.is_cuda:
        return _cuda_listed().listed_mixer(x, lw, spec, ropes, meta, kv, kv_layer, state_layer, eps, carry)
    z = linear(x, lw.wqkv)
    a, r, d, outs = spec.attention, spec.retention, spec.delta, []
    sl, sr = spec.branch_scales if lw.out_norms is None else (1.0, 1.0)
    if a is not None and a.joint_scores:
        q = ref.joint_prep(z[:, : a.qkv_dim], a, meta, kv, kv_layer, eps)
        o = ref.joint_attention(q, kv, kv_layer, meta, a, lw.score_bias, lw.score_mix, lw.sink, eps)
        outs.append(o.reshape(x.shape[0], -1) * sl)
    elif a is not None:
        q = ref.head_prep(z[:, : a.qkv_dim], lw.q_norm, lw.k_norm, a, ropes[0], meta, kv, kv_layer, eps, *first_values(z, a, lw, carry))
        o = ref.paged_attention(q, kv, kv_layer, meta, a.scale, a.window, sink=lw.sink)
        if a.gate:
            o = ref.head_gate(o, z[:, a.qkv_dim : a.proj_dim], a)
        outs.append(o.reshape(x.shape[0], -1) * sl)
    zr = z[:, 0 if a is None else a.proj_dim :]
    if r is not None:
        outs.append((ref.retention(zr, r, ropes[1], meta, kv.states.data[state_layer], eps) * sr).to(x.dtype))
    if d is not None:
        o = ref.delta_rule(zr, lw.delta, d, meta, kv.states.data[state_layer], kv.states.windows[state_layer], eps)
        outs.append((o * sr).to(x.dtype))
    return tuple(outs) if lw.out_norms is not None else torch.cat(outs, dim=-1)


@instrument("gated_ffn")
def gated_ffn(x, gate_up, down):
    """W_down (silu(W_gate x) * (W_up x)) with gate | up as one matrix."""
    if x.is_cuda:
        return _cuda_listed().gated_ffn(x, gate_up, down)
    return linear(silu_mul(linear(x, gate_up)), down)


@instrument("moe_ffn")
def moe_ffn(x, lw, spec, combine=True):
    """Routed experts (``spec``: ``models.config.MoESpec``) with float32 router logits, plus the shared expert.  ``combine``
    False: the result may be ``RoutedRows`` (``joint_norm`` takes either)."""
    if x.is_cuda:
        return _cuda_listed().moe_ffn(x, lw, spec, combine)
    ids, wts = ref.moe_route(linear(x.float(), lw.router), spec, lw.router_bias if spec.correction else None)
    one = gated_ffn if spec.expert.gated else lambda h, up, down: linear(ref.activation(linear(h, up), spec.expert.act), down)
    ex, H = lw.experts, x.shape[1]
    xp = torch.nn.functional.pad(x, (0, ex.gate_up[0].shape[1] - H))
    out = torch.zeros(x.shape[0], ex.down[0].shape[0], dtype=torch.float32)
    for e in range(spec.n_experts):
        rows, slot = (ids == e).nonzero(as_tuple=True)
        if rows.numel():
            y = one(xp[rows], ex.gate_up[e], ex.down[e]).float()
            out.index_add_(0, rows, y * wts[rows, slot][:, None])
    out = out[:, :H]
    if lw.shared_gate_up is not None:
        out = out + gated_ffn(x, lw.shared_gate_up, lw.shared_down).float()
    return out.to(x.dtype)


@instrument("qk_rope_kv_write")
def qk_rope_kv_write(qkv, positions, slot_mapping, kv, layer, rope, q_norm=None, k_norm=None, eps=1e-6, norm_after=False):
    """Split fused qkv [T, (nq+2nkv)*hd], optional per-head QK RMSNorm, RoPE on q and k,
    write K/V into the paged cache.  Returns rotated q as [T, nq, hd].  ``norm_after``: the norms act on the rotated
    vectors (Hunyuan); that order runs as torch operations on either device."""
    norm_after = norm_after and q_norm is not None
    if qkv.is_cuda and not norm_after:
        return _cuda().qk_rope_kv_write(qkv, positions, slot_mapping, kv, layer, rope, q_norm, k_norm, eps)
    nq, nkv, hd = rope.n_heads, rope.n_kv_heads, rope.head_dim
    T = qkv.shape[0]
    q = qkv[:, : nq * hd].reshape(T, nq, hd)
    k = qkv[:, nq * hd : (nq + nkv) * hd].reshape(T, nkv, hd)
    v = qkv[:, (nq + nkv) * hd :].reshape(T, nkv, hd)
    if q_norm is not None and not norm_after:
        q = ref.rmsnorm(q, q_norm, eps)
        k = ref.rmsnorm(k, k_norm, eps)
    q = ref.apply_rope(q, positions, rope.inv_freq, rope.pairing, rope.mscale)
    k = ref.apply_rope(k, positions, rope.inv_freq, rope.pairing, rope.mscale)
    if norm_after:
        q = ref.rmsnorm(q, q_norm, eps).to(qkv.dtype)
        k = ref.rmsnorm(k, k_norm, eps).to(qkv.dtype)
    ref.kv_write(kv, layer, k, v, slot_mapping)
    return q


@instrument("paged_attention")
def paged_attention(q, kv, layer, meta, scale, sliding_window=0, softcap=0.0):
    if q.is_cuda:
        return _cuda().paged_attention(q, kv, layer, meta, scale, sliding_window, softcap=softcap)
    return ref.paged_attention(q, kv, layer, meta, scale, sliding_window, softcap)


@instrument("residual_norm")
def residual_norm(res, y, alpha, w, b, eps, kind="layer", act_dtype=torch.float32, keep_stream=True):
    """norm(alpha * res + y) computed in float32: (the new float32 stream, the same in ``act_dtype``).  ``res`` (float32) or
    ``y`` may be None; without ``keep_stream`` the caller wants the second result only."""
    if w.is_cuda:
        return _cuda_latent().residual_norm(res, y, alpha, w, b, eps, kind, act_dtype, keep_stream)
    return ref.residual_norm(res, y, alpha, w, b, eps, kind, act_dtype)


@instrument("linear_act")
def linear_act(x, w, act):
    """act(x @ W^T): the up projection of a feed-forward block without a gate."""
    if x.is_cuda:
        return _cuda_latent().linear_act(x, w, act)
    return ref.activation(linear(x, w), act)


@instrument("latent_mixer")
def latent_mixer(x, m, spec, rope, meta, kv, layer, eps):
    """Latent attention of one layer up to (not including) its output projection: [T, heads * v_dim].  ``m`` holds the
    projections (``models.weights.MLAWeights``), ``spec`` the geometry (``models.config.LatentAttentionSpec``); the cache
    layer receives this step's rows unless the layer reads another layer's."""
    if x.is_cuda:
        return _cuda_latent().latent_mixer(x, m, spec, rope, meta, kv, layer, eps)
    qkv = linear(x, m.q)
    q = ref.latent_rows(qkv, m, spec, rope, meta, kv, layer, eps)
    o = ref.latent_attention(q, kv, layer, meta, spec.scale, spec.kv_rank, spec.window, m.sink)
    return torch.einsum("thc,hvc->thv", o.float(), m.w_uv.float()).to(x.dtype).reshape(x.shape[0], -1)


@instrument("moe_route")
def moe_route(logits, cfg, bias=None):
    if logits.is_cuda:
        return _cuda().moe_route(logits, cfg, bias)
    return ref.moe_route(logits, cfg, bias)


@instrument("argmax")
def argmax(logits, tie="lowest"):
    if logits.is_cuda:
        return _cuda().argmax(logits, tie)
    return ref.argmax(logits, tie)
