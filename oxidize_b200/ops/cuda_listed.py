"""Bindings of the kernels behind listed layers with grouped-query attention, retention, norms on both sides of a branch and
gated or routed feed-forward blocks (``csrc/oxb_listed.cu``), in bfloat16 and float32.  CUDA tensors only; see
:mod:`oxidize_b200.ops` for the operators' meaning."""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from ..models.config import HEAD_WIDTHS, ROW_TAIL
from . import cuda as opcuda
from . import cuda_latent as latent
from .cuda import _check, _p, _stream

_declared = False

DT = latent.DT


def lib():
    global _declared
    L = latent.lib()
    if not _declared:
        vp, i32, f32 = ctypes.c_void_p, ctypes.c_int, ctypes.c_float
        L.oxb_branch_norm.argtypes = [vp] * 6 + [i32] * 3 + [f32, vp]
        L.oxb_head_prep.argtypes = ([vp, i32, i32, vp, vp, vp] + [i32] * 3 + [vp, vp, i32, f32] + [i32] * 5 + [vp, vp, i32, i32]
                                    + [f32, f32, vp, i32, i32, i32, vp, i32, i32, i32, vp])
        L.oxb_add_normed.argtypes = [vp, vp, i32, vp, vp, i32, vp, i32, f32, vp, vp, i32, vp, vp, vp, i32, i32, i32, vp]
        L.oxb_joint_norm.argtypes = [vp] * 5 + [f32, f32, vp, i32, vp, vp, i32, vp, vp, vp] + [i32] * 3 + [f32, vp]
        L.oxb_gqa_attention_simt.argtypes = [vp, vp, i32, f32, vp, i32, vp, vp, vp, vp] + [i32] * 9 + [f32, vp, i32, i32, vp]
        L.oxb_kv_gather.argtypes = [vp] * 4 + [i32] * 7 + [vp, vp]
        L.oxb_gqa_prefill.argtypes = [vp, vp, vp, i32, f32] + [vp] * 5 + [i32] * 7 + [f32, i32, vp, i32, i32, vp]
        L.oxb_retention_chunk_supported.argtypes = L.oxb_retention_mma_supported.argtypes = [i32, i32]
        L.oxb_retention.argtypes = ([vp, i32, i32] + [vp] * 4 + [i32] * 3 + [vp, vp, i32, vp, i32, f32] + [i32] * 5 + [f32, f32]
                                    + [i32] * 4 + [vp, vp])
        L.oxb_silu_mul_f32.argtypes = [vp, vp, vp, i32, i32, vp]
        L.oxb_moe_combine_f32.argtypes = [vp, i32, vp, vp, i32, vp, vp, i32, i32, vp]
        L.oxb_router_logits.argtypes = [vp, vp, i32, vp] + [i32] * 3 + [vp]
        L.oxb_gemm_f32_rows.argtypes = [vp] * 5 + [i32] * 7 + [vp]
        _declared = True
    return L


# --------------------------------------------------------------------------- norms
def branch_norm(res: torch.Tensor, y: Optional[torch.Tensor], w_post: Optional[torch.Tensor], w_next: Optional[torch.Tensor],
                eps: float, act_dtype: torch.dtype):
    T, H = res.shape
    if y is not None and (y.dtype != act_dtype or not y.is_contiguous()):
        y = y.to(act_dtype).contiguous()
    x = res if y is None else torch.empty_like(res)
    a = None if w_next is None else torch.empty(T, H, dtype=act_dtype, device=res.device)
    _check(lib().oxb_branch_norm(res.data_ptr(), _p(y), _p(w_post), _p(w_next), None if y is None else x.data_ptr(), _p(a),
                                 DT[act_dtype], T, H, eps, _stream()), "oxb_branch_norm")
    return x, a


def joint_norm(res: torch.Tensor, mix, ffn, w_next: Optional[torch.Tensor], eps: float, act_dtype: torch.dtype):
    from . import NormedPair, RoutedRows

    T, H = res.shape

    def rows(t):
        return t if t is None or (t.dtype == act_dtype and t.is_contiguous()) else t.to(act_dtype).contiguous()

    pair = mix if isinstance(mix, NormedPair) else None
    y0, y1 = (rows(pair.left), rows(pair.right)) if pair else (rows(mix), None)
    routed = ffn if isinstance(ffn, RoutedRows) else None
    f = rows(routed.rows if routed else ffn)
    x = res if mix is None and ffn is None else torch.empty_like(res)
    a = None if w_next is None else torch.empty(T, H, dtype=act_dtype, device=res.device)
    _check(lib().oxb_joint_norm(res.data_ptr(), _p(y0), _p(y1), _p(pair.left_norm) if pair else None, _p(pair.right_norm) if pair else None,
                                pair.left_scale if pair else 1.0, pair.right_scale if pair else 1.0, _p(f), 0 if f is None else f.stride(0),
                                _p(routed.index) if routed else None, _p(routed.weights) if routed else None,
                                routed.index.shape[1] if routed else 0, _p(w_next), None if x is res else x.data_ptr(), _p(a),
                                DT[act_dtype], T, H, eps, _stream()), "oxb_joint_norm")
    return x, a


def add_normed(res: torch.Tensor, y, w: torch.Tensor, groups: int, eps: float, act_dtype: Optional[torch.dtype], streams=None,
               depth: Optional[torch.Tensor] = None):
    from . import RoutedRows

    T, H = res.shape
    routed = y if isinstance(y, RoutedRows) else None
    f = routed.rows if routed else y
    if f.stride(-1) != 1:
        f = f.contiguous()
    x = torch.empty_like(res)
    # (a float32 activation is the stream itself)
    a = x if act_dtype == torch.float32 else None if act_dtype is None else torch.empty(T, H, dtype=act_dtype, device=res.device)
    first = results = None
    n = 0
    if streams is not None:
        first, results, n = streams.first, streams.results, streams.n
        streams.n += 1
    _check(lib().oxb_add_normed(res.data_ptr(), f.data_ptr(), f.stride(0), _p(routed.index) if routed else None,
                                _p(routed.weights) if routed else None, routed.index.shape[1] if routed else 0, w.data_ptr(), groups, eps,
                                _p(first), _p(results), n, _p(depth) if streams is not None else None, x.data_ptr(),
                                None if a is x else _p(a), DT[f.dtype], T, H, _stream()), "oxb_add_normed")
    return x, a


def grouped_norm(x: torch.Tensor, w: torch.Tensor, groups: int, eps: float, act_dtype: torch.dtype) -> torch.Tensor:
    T, H = x.shape
    x = x.contiguous()
    a = torch.empty(T, H, dtype=act_dtype, device=x.device)
    _check(lib().oxb_add_normed(x.data_ptr(), None, H, None, None, 0, w.data_ptr(), groups, eps, None, None, 0, None, None, a.data_ptr(),
                                DT[act_dtype], T, H, _stream()), "oxb_add_normed")
    return a


# --------------------------------------------------------------------------- attention
def head_prep(z: torch.Tensor, q_norm, k_norm, spec, rope, meta, kv, layer: int, eps: float, v_first: Optional[torch.Tensor] = None,
              v_mix: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q | k | v projections [T, ...] to (rotated, scaled) queries [T, heads, width]; keys and (mixed) values go into the cache
    pages."""
    T = z.shape[0]
    tab = meta.positions if rope is None else opcuda.rope_table(rope, rope.max_pos)  # (nothing of it is read without a rotation)
    max_pos, rot, pairing = (1, 0, 0) if rope is None else (tab.shape[0], tab.shape[1], 0 if rope.pairing == "split_half" else 1)
    first = (None, 0, 0) if v_first is None else (v_first.data_ptr(), v_first.stride(0), v_first.shape[2])
    q = torch.empty(T, spec.heads, spec.width, dtype=z.dtype, device=z.device)
    _check(lib().oxb_head_prep(z.data_ptr(), z.stride(0), DT[z.dtype], meta.positions.data_ptr(), meta.slot_mapping.data_ptr(),
                               tab.data_ptr(), max_pos, rot, pairing, _p(q_norm), _p(k_norm), 1 if spec.qk_norm == "full" else 0, eps, T, spec.heads, spec.kv_heads, spec.dim,
                               spec.width, q.data_ptr(), kv.data[layer].data_ptr(), kv.page_size, kv.num_blocks, spec.temp_coef, spec.temp_every,
                               *first, spec.v_dim, _p(v_mix), int(spec.qk_norm == "unit"), int(spec.shared_kv),
                               ROW_TAIL if spec.shared_kv else 0, _stream()), "oxb_head_prep")
    return q


def _gate(gate: Optional[torch.Tensor], spec):
    return (None, 0, 0) if gate is None else (gate.data_ptr(), gate.stride(0), int(spec.gate == "value"))


def attention_simt(q, kv, layer: int, meta, spec, sink, out, out_scale: float, gate=None) -> None:
    T, H, W = q.shape
    B = meta.seq_lens.shape[0]
    _check(lib().oxb_gqa_attention_simt(q.data_ptr(), out.data_ptr(), out.stride(0), out_scale, kv.data[layer].data_ptr(), DT[q.dtype],
                                        meta.block_tables.data_ptr(), meta.seq_lens.data_ptr(), meta.query_start.data_ptr(), _p(sink),
                                        B, meta.block_tables.stride(0), T, H, spec.kv_heads, W, kv.page_size, kv.num_blocks,
                                        spec.window, spec.scale, *_gate(gate, spec), _stream()), "oxb_gqa_attention_simt")


def attention_prefill(q, kv, layer: int, meta, spec, sink, out, out_scale: float, gate=None) -> None:
    """Long portions: the visible rows are gathered from their pages, then flash attention on tcgen05."""
    T, H, W = q.shape
    B, G = meta.seq_lens.shape[0], spec.kv_heads
    lo, off, rows = latent._spans(meta, spec.window)
    dense = torch.empty(rows, 2 * G * W, dtype=q.dtype, device=q.device)
    _check(lib().oxb_kv_gather(kv.data[layer].data_ptr(), meta.block_tables.data_ptr(), lo.data_ptr(), off.data_ptr(), B, rows,
                               meta.block_tables.stride(0), G, W, kv.page_size, kv.num_blocks, dense.data_ptr(), _stream()),
           "oxb_kv_gather")
    _check(lib().oxb_gqa_prefill(q.data_ptr(), dense.data_ptr(), out.data_ptr(), out.stride(0), out_scale, meta.query_start.data_ptr(),
                                 meta.seq_lens.data_ptr(), lo.data_ptr(), off.data_ptr(), _p(sink), B, T, H, G, rows, W, spec.window,
                                 spec.scale, max(n for n, _ in meta.host_lens), *_gate(gate, spec), _stream()), "oxb_gqa_prefill")


def attention(q, kv, layer: int, meta, spec, sink, out, out_scale: float, gate: Optional[torch.Tensor] = None) -> None:
    """Attention of a step's queries over the cache into ``out`` [T, heads * width] (may be a column slice), times the sigmoid of
    ``gate`` ([T, heads or more], or [T, heads * width] with a gate per value)."""
    if q.dtype != torch.bfloat16 or kv.page_size != 16 or spec.width not in HEAD_WIDTHS:
        attention_simt(q, kv, layer, meta, spec, sink, out, out_scale, gate)
        return

    def paged(qs, sub, o, gs) -> None:
        opcuda.paged_attention(qs, kv, layer, sub, spec.scale, spec.window, sink=sink, out=o, out_scale=out_scale, gate=gs,
                               gate_per_value=spec.gate == "value")

    if (not meta.host_lens or max(n for n, _ in meta.host_lens) < latent.EXPAND_ROWS
            or not lib().oxb_latent_prefill_supported(spec.width, 0, spec.width)
            or latent._spans(meta, spec.window)[2] > latent.MAX_SPAN):
        paged(q, meta, out, gate)
        return
    starts = [0]
    for n, _ in meta.host_lens:
        starts.append(starts[-1] + n)
    runs = latent._runs(meta.host_lens)
    for b0, b1, big in runs:
        t0, t1 = starts[b0], starts[b1]
        sub = meta if len(runs) == 1 else latent._sub_batch(meta, b0, b1, t0, t1)
        gs = None if gate is None else gate[t0:t1]
        if big:
            attention_prefill(q[t0:t1], kv, layer, sub, spec, sink, out[t0:t1], out_scale, gs)
        else:
            paged(q[t0:t1], sub, out[t0:t1], gs)


# --------------------------------------------------------------------------- retention
CHUNK_ROWS = 9  # sequences that feed at least this many rows in a step go through chunks on the tensor cores
SEGMENT_ROWS = 256  # a segment of a long portion is at least this long
_ALL = 1 << 30


def segments(rows: int, seqs: int, heads: int, sms: int) -> int:
    """Segments of the longest portion: as many as keep one CTA per SM busy."""
    return max(1, min(rows // SEGMENT_ROWS, sms // max(1, seqs * heads), 32))


def chunk_form(K: int, V: int) -> int:
    """Which kernel takes long portions: 2 tcgen05, 1 mma.sync (wider keys), 0 neither (the token-by-token kernel does)."""
    L = lib()
    return 2 if L.oxb_retention_mma_supported(K, V) else 1 if L.oxb_retention_chunk_supported(K, V) else 0


def retention(z: torch.Tensor, spec, rope, meta, state: torch.Tensor, decay: torch.Tensor, eps: float, out: torch.Tensor,
              out_scale: float, chunk_rows: Optional[int] = None, n_seg: Optional[int] = None, form: Optional[int] = None) -> None:
    """z [T, q | k | v | gate] to the normed, gated heads ``out`` [T, heads * v_width]; ``state`` [slots, H, K, V] is updated."""
    L = lib()
    H, K, V = spec.state_shape
    B = meta.seq_lens.shape[0]
    tab = opcuda.rope_table(rope, rope.max_pos)
    if meta.state_slots is None:
        raise ValueError("a layer with a recurrent state needs the sequences' state slots")

    def run(lo: int, hi: int, chunk: int, seg: int, ws) -> None:
        _check(L.oxb_retention(z.data_ptr(), z.stride(0), DT[z.dtype], meta.query_start.data_ptr(), meta.seq_lens.data_ptr(),
                               meta.state_slots.data_ptr(), tab.data_ptr(), tab.shape[0], tab.shape[1],
                               0 if rope.pairing == "split_half" else 1, decay.data_ptr(), state.data_ptr(), state.shape[0],
                               out.data_ptr(), out.stride(0), out_scale, B, H, K, V, spec.v_dim, spec.dim ** -0.5, eps, lo, hi, chunk,
                               seg, _p(ws), _stream()), "oxb_retention")

    most = max(1, meta.max_query_len)
    least = 1 if meta.host_lens is None else min(n for n, _ in meta.host_lens)
    cut = CHUNK_ROWS if chunk_rows is None else chunk_rows
    if form is None:
        form = chunk_form(K, V)
    if z.dtype != torch.bfloat16 or most < cut or form == 0:
        run(1, _ALL, 0, 1, None)
        return
    if least < cut:
        run(1, cut - 1, 0, 1, None)
    if n_seg is None:
        seqs = B if meta.host_lens is None else sum(n >= cut for n, _ in meta.host_lens)
        n_seg = segments(most, seqs, H, opcuda.sm_count(z.device))
    block = 128 * 128 if form == 2 else K * V  # floats of a segment's block
    ws = torch.empty(B * H * n_seg * block, dtype=torch.float32, device=z.device) if n_seg > 1 else None
    run(cut, _ALL, form, n_seg, ws)


def listed_mixer(x: torch.Tensor, lw, spec, ropes, meta, kv, kv_layer: int, state_layer: int, eps: float, carry=None):
    from . import first_values, linear

    z = linear(x, lw.wqkv)
    a, r, d = spec.attention, spec.retention, spec.delta
    apart = lw.out_norms is not None  # each side has an output projection (and a scale) of its own
    sl, sr = (1.0, 1.0) if apart else spec.branch_scales
    T = x.shape[0]
    outs = [torch.empty(T, n, dtype=x.dtype, device=x.device) for n in ((a.out_dim, spec.recurrent.out_dim) if apart else (spec.out_dim,))]
    na = no = 0
    if a is not None:
        if kv.data[kv_layer].dtype != x.dtype:
            raise ValueError(f"cache rows of listed layers are kept in the compute type on the GPU ({x.dtype}), not {kv.dtype_name}")
        na, no = a.proj_dim, a.out_dim
        prep = () if a.joint_scores else first_values(z, a, lw, carry)
        q = head_prep(z[:, : a.qkv_dim], lw.q_norm, lw.k_norm, a, ropes[0], meta, kv, kv_layer, eps, *prep)
        if a.joint_scores:
            from . import cuda_joint

            cuda_joint.attention(q, kv, kv_layer, meta, a, lw.score_bias, lw.score_mix, lw.sink, outs[0][:, :no], sl)
        else:
            attention(q, kv, kv_layer, meta, a, lw.sink, outs[0][:, :no], sl, z[:, a.qkv_dim : na] if a.gate else None)
    out = outs[-1][:, 0 if apart else no :]
    if d is not None:
        from . import cuda_delta

        cuda_delta.delta_rule(z[:, na:], lw.delta, d, meta, kv.states.data[state_layer], kv.states.windows[state_layer], eps, out, sr)
    if r is not None:
        decay = getattr(lw, "_decay", None)
        if decay is None:
            decay = lw._decay = torch.tensor(r.decay, dtype=torch.float32, device=x.device)
        retention(z[:, na:], r, ropes[1], meta, kv.states.data[state_layer], decay, eps, out, sr)
    return tuple(outs) if apart else outs[0]


# --------------------------------------------------------------------------- feed-forward blocks
def silu_mul_f32(gu: torch.Tensor, n_rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    T, F2 = gu.shape
    out = torch.empty(T, F2 // 2, dtype=torch.float32, device=gu.device)
    _check(lib().oxb_silu_mul_f32(gu.data_ptr(), out.data_ptr(), _p(n_rows), T, F2 // 2, _stream()), "oxb_silu_mul_f32")
    return out


def gated_ffn(x: torch.Tensor, gate_up, down) -> torch.Tensor:
    from . import linear

    if x.dtype == torch.float32:
        return linear(silu_mul_f32(linear(x, gate_up)), down)
    if gate_up.swiglu_interleaved:
        xp, data = opcuda.pad_k(x.contiguous(), gate_up.parts[0])
        return linear(opcuda.linear_swiglu(xp, data), down)
    return linear(opcuda.silu_mul(linear(x, gate_up)), down)


def router_logits(x: torch.Tensor, w) -> torch.Tensor:
    """[T, experts] float32, never rounded to 16 bits."""
    x = x.contiguous()
    T, K = x.shape
    out = torch.empty(T, w.shape[0], dtype=torch.float32, device=x.device)
    if w.data.dtype != x.dtype:
        raise ValueError(f"router weights are kept in the compute type ({x.dtype}), not {w.data.dtype}")
    _check(lib().oxb_router_logits(x.data_ptr(), w.data.data_ptr(), DT[x.dtype], out.data_ptr(), T, w.shape[0], K, _stream()),
           "oxb_router_logits")
    return out


def _gemm_rows(x, w, offsets, perm, groups: int, rows: int, max_rows: int, act: int = 0) -> torch.Tensor:
    N, K = w.shape[0] // groups, w.shape[1]
    y = torch.empty(rows, N, dtype=torch.float32, device=x.device)
    _check(lib().oxb_gemm_f32_rows(x.data_ptr(), w.data.data_ptr(), y.data_ptr(), offsets.data_ptr(), _p(perm), groups, max_rows, N, K,
                                   x.stride(0), N, act, _stream()), "oxb_gemm_f32_rows")
    return y


def moe_ffn(x: torch.Tensor, lw, spec, combine: bool = True):
    from . import RoutedRows, cuda_moe

    T, H = x.shape
    ex = lw.experts
    bias = lw.router_bias if spec.correction else None
    relu2 = not spec.expert.gated
    if relu2 and spec.expert.act != "relu2":
        raise ValueError(f"ungated experts have the relu2 activation, not {spec.expert.act!r}")
    logits = router_logits(x, lw.router)
    shared = gated_ffn(x, lw.shared_gate_up, lw.shared_down) if lw.shared_gate_up is not None else None
    pad = ex.gate_up_stack.shape[1] - H
    xp = torch.nn.functional.pad(x, (0, pad)) if pad else x.contiguous()
    if x.dtype == torch.bfloat16:
        sp = torch.nn.functional.pad(shared, (0, pad)) if pad and shared is not None else shared
        if not combine and shared is None and T * spec.n_experts_used <= cuda_moe.MAX_DISPATCH_ENTRIES:
            return RoutedRows(*cuda_moe.moe_layer(xp, logits, spec, bias, ex, relu2=relu2, combine=False))
        out = cuda_moe.moe_layer(xp, logits, spec, bias, ex, sp, relu2=relu2)[0]
        return out[:, :H].contiguous() if pad else out
    E, k = spec.n_experts, spec.n_experts_used
    if E > 256 or T * k > cuda_moe.MAX_DISPATCH_ENTRIES:
        raise ValueError("float32 expert dispatch covers up to 256 experts and 2^17 token x expert pairs in a step")
    ids, wts = cuda_moe.moe_route(logits, spec, bias)
    offsets, perm, inv = cuda_moe.moe_dispatch(ids, 0, E)
    h = _gemm_rows(xp, ex.gate_up_stack, offsets, perm, E, T * k, T, latent.ACTS["relu2"] if relu2 else 0)
    y = _gemm_rows(h if relu2 else silu_mul_f32(h, offsets[E:]), ex.down_stack, offsets, None, E, T * k, T)
    if not combine and shared is None:
        return RoutedRows(y, inv, wts)
    out = torch.empty(T, H, dtype=torch.float32, device=x.device)
    _check(lib().oxb_moe_combine_f32(y.data_ptr(), y.stride(0), inv.data_ptr(), wts.data_ptr(), k, _p(shared), out.data_ptr(), T, H,
                                     _stream()), "oxb_moe_combine_f32")
    return out
