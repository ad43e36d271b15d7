"""Bindings of the kernels behind models with latent attention and norms after the sum (``csrc/oxb_latent.cu``), and of the
float32 compute path.  CUDA tensors only; see :mod:`oxidize_b200.ops` for the operators' meaning."""
from __future__ import annotations

import ctypes
from typing import Optional, Sequence

import torch

from . import cuda as opcuda
from .cuda import _check, _p, _stream

_declared = False

DT = {torch.float32: 0, torch.bfloat16: 2}
ACTS = {"relu2": 1}
EPI_RELU2 = 5


def lib():
    global _declared
    L = opcuda.lib()
    if not _declared:
        vp, i32, f32, i64 = ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_longlong
        L.oxb_residual_norm.argtypes = [vp, vp, f32, vp, vp, vp, vp, i32, i32, i32, f32, i32, vp]
        L.oxb_gemm_f32.argtypes = [vp, vp, vp, vp] + [i32] * 7 + [i64, i64, i64, i32, vp]
        L.oxb_latent_prep.argtypes = ([vp, i32, i32, vp, vp, vp, i32, i32, i32, vp, f32] + [i32] * 6 + [vp, i32, vp, vp, i32, i32,
                                      vp, i32, i32, vp])
        L.oxb_latent_attention_simt.argtypes = [vp, vp, vp, i32, vp, vp, vp, vp] + [i32] * 9 + [f32, vp]
        L.oxb_latent_mma_supported.argtypes = [i32] * 3
        L.oxb_latent_attention_mma.argtypes = [vp] * 7 + [i32] * 9 + [f32] + [i32] * 2 + [vp]
        L.oxb_latent_gather.argtypes = [vp] * 4 + [i32] * 7 + [vp] * 3
        L.oxb_latent_prefill_supported.argtypes = [i32] * 3
        L.oxb_latent_prefill.argtypes = [vp] * 9 + [i32] * 12 + [f32, i32, vp]
        L.oxb_gemm_batched.argtypes = [vp, vp, vp, i64] + [i32] * 5 + [vp]
        _declared = True
    return L


# --------------------------------------------------------------------------- norms and products
def residual_norm(res: Optional[torch.Tensor], y: Optional[torch.Tensor], alpha: float, w: torch.Tensor,
                  b: Optional[torch.Tensor], eps: float, kind: str, act_dtype: torch.dtype, keep_stream: bool = True):
    like = y if res is None else res
    T, H = like.shape
    if y is not None and (y.dtype != act_dtype or not y.is_contiguous()):
        y = y.to(act_dtype).contiguous()
    x = torch.empty(T, H, dtype=torch.float32, device=like.device) if keep_stream or act_dtype == torch.float32 else None
    a = x if act_dtype == torch.float32 else torch.empty(T, H, dtype=act_dtype, device=like.device)
    _check(lib().oxb_residual_norm(_p(res), _p(y), alpha, w.data_ptr(), _p(b), _p(x), None if a is x else a.data_ptr(),
                                   DT[act_dtype], T, H, eps, 1 if kind == "layer" else 0, _stream()), "oxb_residual_norm")
    return x, a


def gemm_f32(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, bias: Optional[torch.Tensor] = None, act: int = 0,
             groups: int = 1, dims=None, strides=(0, 0, 0)) -> torch.Tensor:
    """out = act(x @ w^T + bias) in float32; grouped calls give (T, N, K, ldx, ldw, ldy) and the group strides."""
    if dims is None:
        T, K = x.shape
        dims = (T, w.shape[0], K, x.stride(0), w.stride(0), out.stride(0))
    _check(lib().oxb_gemm_f32(x.data_ptr(), w.data_ptr(), out.data_ptr(), _p(bias), *dims, groups, *strides, act, _stream()),
           "oxb_gemm_f32")
    return out


def linear_f32(x: torch.Tensor, parts: Sequence, bias: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None,
               act: int = 0) -> torch.Tensor:
    x = x.contiguous()
    if out is None:
        out = torch.empty(x.shape[0], sum(p.shape[0] for p in parts), dtype=torch.float32, device=x.device)
    off = 0
    for p in parts:
        n = p.shape[0]
        gemm_f32(x, p.data, out[:, off : off + n], None if bias is None else bias[off : off + n], act)
        off += n
    return out


def linear_act(x: torch.Tensor, w, act: str) -> torch.Tensor:
    """act(x W^T): the activation is the product's epilogue."""
    p = w.parts[0]
    if x.dtype == torch.float32:
        return linear_f32(x, w.parts, w.bias, act=ACTS[act])
    if act != "relu2" or len(w.parts) != 1 or w.bias is not None or p.qtype != "BF16":
        raise ValueError("linear_act covers one bfloat16 matrix and the relu2 activation")
    x, data = opcuda.pad_k(x.contiguous(), p)
    return opcuda.gemm_bf16(x, data, epi=EPI_RELU2)


# --------------------------------------------------------------------------- latent attention
class LatentOperands:
    """A layer's per-head up-projections in the shapes the products read: ``k`` [H * rank, nope (padded)] multiplies the
    queries (W_uk transposed per head), ``v`` [H * v_dim, latent_pad] the attended latents."""

    def __init__(self, m, spec, dtype: torch.dtype):
        H = m.w_uk.shape[0]
        ld = (spec.nope_dim + 7) // 8 * 8
        dev = m.w_uk.device
        k = torch.zeros(H, spec.kv_rank, ld, dtype=dtype, device=dev)
        k[:, :, : spec.nope_dim] = m.w_uk.transpose(1, 2)
        v = torch.zeros(H, spec.v_dim, spec.latent_pad, dtype=dtype, device=dev)
        v[:, :, : spec.kv_rank] = m.w_uv
        self.heads, self.nope_ld, self.k, self.v = H, ld, k, v
        # expanded form: one matrix that turns a latent into every head's key part and value
        self.v_ld, self.v_off = (spec.v_dim + 7) // 8 * 8, H * ld
        self.kv_ld = H * (ld + self.v_ld)
        self.expand = None
        if dtype == torch.bfloat16:
            e = torch.zeros(self.kv_ld, spec.latent_pad, dtype=dtype, device=dev)
            e[: self.v_off].view(H, ld, -1)[:, : spec.nope_dim, : spec.kv_rank] = m.w_uk
            e[self.v_off :].view(H, self.v_ld, -1)[:, : spec.v_dim, : spec.kv_rank] = m.w_uv
            self.expand = e


def operands(m, spec, dtype: torch.dtype) -> LatentOperands:
    op = getattr(m, "_operands", None)
    if op is None:
        op = m._operands = LatentOperands(m, spec, dtype)
    return op


def batched(x: torch.Tensor, w: torch.Tensor, y: torch.Tensor, y_stride: int, ldy: int) -> None:
    """For every head g: y[:, g * y_stride : g * y_stride + N] = x[g] @ w[g]^T, x [H, T, K], w [H, N, K], rows of y ``ldy``
    apart."""
    H, T, K = x.shape
    N = w.shape[1]
    if x.dtype == torch.float32:
        gemm_f32(x, w, y, groups=H, dims=(T, N, K, K, K, ldy), strides=(T * K, N * K, y_stride))
        return
    _check(lib().oxb_gemm_batched(x.data_ptr(), w.data_ptr(), y.data_ptr(), y_stride, H, T, N, K, ldy, _stream()),
           "oxb_gemm_batched")


def latent_prep(qkv, m, spec, rope, meta, kv, layer: int, eps: float, op: LatentOperands, q_nope=None, q_rows=None, q_full=None):
    tab = opcuda.rope_table(rope, rope.max_pos)
    own = spec.kv_from is None
    _check(lib().oxb_latent_prep(qkv.data_ptr(), qkv.stride(0), DT[qkv.dtype], meta.positions.data_ptr(),
                                 meta.slot_mapping.data_ptr() if own else None, tab.data_ptr(), tab.shape[0], spec.rope_dim,
                                 0 if rope.pairing == "split_half" else 1, _p(m.kv_a_norm), eps, qkv.shape[0], op.heads,
                                 spec.nope_dim, spec.kv_rank, spec.latent_pad, spec.row_dim, _p(q_nope), op.nope_ld, _p(q_rows),
                                 _p(q_full), 0 if q_full is None else q_full.shape[-1], (spec.nope_dim + 15) // 16 * 16, kv.data[layer].data_ptr(), kv.page_size,
                                 kv.num_blocks, _stream()), "oxb_latent_prep")


def attention_simt(q, kv, layer: int, meta, spec, sink, out):
    T, H, width = q.shape
    B = meta.seq_lens.shape[0]
    _check(lib().oxb_latent_attention_simt(q.data_ptr(), out.data_ptr(), kv.data[layer].data_ptr(), DT[q.dtype],
                                           meta.block_tables.data_ptr(), meta.seq_lens.data_ptr(), meta.query_start.data_ptr(),
                                           _p(sink), B, meta.block_tables.stride(0), T, H, spec.latent_pad, width, kv.page_size,
                                           kv.num_blocks, spec.window, spec.scale, _stream()), "oxb_latent_attention_simt")


def mma_splits(B: int, row_blocks: int, window: int, max_len: int, sms: int, most: int) -> int:
    """Key splits of the tensor-core kernel: as many as fit one wave of CTAs (one per SM), a 128-key tile or more each; the
    splits of a row block are one cluster of at most ``most`` CTAs (more than eight only where they fill few clusters)."""
    span = min(window, max_len) if window > 0 else max_len
    tiles = span // 128 + 1
    if B * row_blocks > 2:
        most = min(most, 8)
    return max(1, min(sms // max(1, B * row_blocks), tiles, most))


def attention_mma(q, kv, layer: int, meta, spec, sink, out, splits: Optional[int] = None):
    """Absorbed-form attention on the tensor cores; False when the kernel does not cover the row's shape."""
    T, H, width = q.shape
    B = meta.seq_lens.shape[0]
    mq = max(1, meta.max_query_len)
    if not lib().oxb_latent_mma_supported(spec.latent_pad, width, kv.page_size):
        return False
    row_blocks = (mq * H + 31) // 32
    if splits is None:
        splits = mma_splits(B, row_blocks, spec.window, meta.max_seq_len or kv.page_size, opcuda.sm_count(q.device),
                            lib().oxb_latent_max_splits())
    _check(lib().oxb_latent_attention_mma(q.data_ptr(), out.data_ptr(), kv.data[layer].data_ptr(), meta.block_tables.data_ptr(),
                                          meta.seq_lens.data_ptr(), meta.query_start.data_ptr(), _p(sink), B,
                                          meta.block_tables.stride(0), T, H, spec.latent_pad, width, kv.page_size, kv.num_blocks,
                                          spec.window, spec.scale, mq, splits, _stream()),
           "oxb_latent_attention_mma")
    return True


def latent_mixer(x, m, spec, rope, meta, kv, layer: int, eps: float) -> torch.Tensor:
    from . import linear

    if kv.data[layer].dtype != x.dtype:
        raise ValueError(f"latent cache rows are kept in the compute type on the GPU ({x.dtype}), not {kv.dtype_name}")
    return latent_core(linear(x, m.q), m, spec, rope, meta, kv, layer, eps, operands(m, spec, x.dtype))


# Sequences that feed at least this many rows in a step take the expanded form; MAX_SPAN bounds the rows expanded at once.
EXPAND_ROWS, MAX_SPAN = 64, 1 << 16


def _spans(meta, window: int):
    """(first visible position of every sequence, its first dense row, total rows) of a step for one window, kept for the
    other layers of the step."""
    key = ("latent_spans", window)
    got = meta.extra.get(key)
    if got is None:
        lo = [max(0, ctx - n - window + 1) if window > 0 else 0 for n, ctx in meta.host_lens]
        off = [0]
        for l, (_, ctx) in zip(lo, meta.host_lens):
            off.append(off[-1] + ctx - l)
        t = torch.tensor(lo + off, dtype=torch.int32, device=meta.seq_lens.device)
        got = meta.extra[key] = (t[: len(lo)], t[len(lo) :], off[-1])
    return got


def latent_expanded(qkv, m, spec, rope, meta, kv, layer: int, eps: float, op: LatentOperands, out: torch.Tensor) -> None:
    """Long portions: keys and values of the visible rows are expanded per head, then flash attention."""
    T, H, dt, dev = qkv.shape[0], op.heads, qkv.dtype, qkv.device
    B = meta.seq_lens.shape[0]
    full = (spec.nope_dim + 15) // 16 * 16 + (spec.row_dim - spec.latent_pad)
    q = torch.empty(T, H, full, dtype=dt, device=dev)
    latent_prep(qkv, m, spec, rope, meta, kv, layer, eps, op, q_full=q)
    lo, off, rows = _spans(meta, spec.window)
    lat = torch.empty(rows, spec.latent_pad, dtype=dt, device=dev)
    rot = torch.empty(rows, spec.row_dim - spec.latent_pad, dtype=dt, device=dev)
    _check(lib().oxb_latent_gather(kv.data[layer].data_ptr(), meta.block_tables.data_ptr(), lo.data_ptr(), off.data_ptr(), B, rows,
                                   meta.block_tables.stride(0), spec.latent_pad, spec.row_dim, kv.page_size, kv.num_blocks,
                                   lat.data_ptr(), rot.data_ptr(), _stream()), "oxb_latent_gather")
    full_kv = opcuda.gemm_bf16(lat, op.expand)
    _check(lib().oxb_latent_prefill(q.data_ptr(), full_kv.data_ptr(), rot.data_ptr(), out.data_ptr(), meta.query_start.data_ptr(),
                                    meta.seq_lens.data_ptr(), lo.data_ptr(), off.data_ptr(), _p(m.sink), B, T, H, rows, spec.nope_dim,
                                    spec.rope_dim, spec.v_dim, op.kv_ld, op.nope_ld, op.v_off, op.v_ld, spec.window, spec.scale,
                                    max(n for n, _ in meta.host_lens), _stream()), "oxb_latent_prefill")


def _runs(lens):
    """Maximal runs [(first, end, long)] of neighbouring sequences that are all long or all short portions."""
    runs = []
    for b, (n, _) in enumerate(lens):
        big = n >= EXPAND_ROWS
        if runs and runs[-1][2] == big:
            runs[-1][1] = b + 1
        else:
            runs.append([b, b + 1, big])
    return runs


def _sub_batch(meta, b0: int, b1: int, t0: int, t1: int):
    """Sequences [b0, b1) (rows [t0, t1)) of a step as a step of their own, kept for the other layers."""
    key = ("latent_sub", b0, b1)
    sub = meta.extra.get(key)
    if sub is None:
        lens = meta.host_lens[b0:b1]
        sub = meta.extra[key] = type(meta)(
            None, meta.positions[t0:t1], meta.slot_mapping[t0:t1], (meta.query_start[b0 : b1 + 1] - t0).contiguous(),
            meta.seq_lens[b0:b1], meta.block_tables[b0:b1], None, max(n for n, _ in lens), max(c for _, c in lens), b1 - b0,
            host_lens=lens)
    return sub


def latent_core(qkv, m, spec, rope, meta, kv, layer: int, eps: float, op: LatentOperands) -> torch.Tensor:
    """From the layer's projections to its heads' outputs [T, heads * v_dim]."""
    T, H, dt, dev = qkv.shape[0], op.heads, qkv.dtype, qkv.device
    out = torch.empty(T, H * spec.v_dim, dtype=dt, device=dev)
    if (dt == torch.bfloat16 and meta.host_lens and any(n >= EXPAND_ROWS for n, _ in meta.host_lens)
            and lib().oxb_latent_prefill_supported(spec.nope_dim, spec.rope_dim, spec.v_dim)
            and _spans(meta, spec.window)[2] <= MAX_SPAN):
        starts = [0]
        for n, _ in meta.host_lens:
            starts.append(starts[-1] + n)
        runs = _runs(meta.host_lens)
        for b0, b1, big in runs:
            t0, t1 = starts[b0], starts[b1]
            sub = meta if len(runs) == 1 else _sub_batch(meta, b0, b1, t0, t1)
            (latent_expanded if big else latent_absorbed)(qkv[t0:t1], m, spec, rope, sub, kv, layer, eps, op, out[t0:t1])
    else:
        latent_absorbed(qkv, m, spec, rope, meta, kv, layer, eps, op, out)
    return out


def latent_absorbed(qkv, m, spec, rope, meta, kv, layer: int, eps: float, op: LatentOperands, out: torch.Tensor) -> None:
    """Decode rows and short portions: attention over the cached rows themselves, W_uk and W_uv applied to the queries and
    to the attended latents."""
    T, H, dt, dev = qkv.shape[0], op.heads, qkv.dtype, qkv.device
    q_nope = torch.empty(H, T, op.nope_ld, dtype=dt, device=dev)
    q = torch.empty(T, H, spec.row_dim, dtype=dt, device=dev)
    latent_prep(qkv, m, spec, rope, meta, kv, layer, eps, op, q_nope=q_nope, q_rows=q)
    batched(q_nope, op.k, q, spec.row_dim, H * spec.row_dim)
    o = torch.empty(H, T, spec.latent_pad, dtype=dt, device=dev)
    if dt != torch.bfloat16 or not attention_mma(q, kv, layer, meta, spec, m.sink, o):
        attention_simt(q, kv, layer, meta, spec, m.sink, o)
    batched(o, op.v, out, spec.v_dim, H * spec.v_dim)
