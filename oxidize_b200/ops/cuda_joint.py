"""Bindings of the attention kernels that work on the scores of all heads together (``csrc/oxb_joint.cu``), in bfloat16 and
float32.  CUDA tensors only; see :func:`oxidize_b200.ops.ref.joint_attention` for the operator's meaning."""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from ..models.config import ROW_TAIL
from . import cuda as opcuda
from . import cuda_latent as latent
from .cuda import _check, _p, _stream

_declared = False
_ALL = 1 << 30
LONG_ROWS = 16  # sequences that feed at least this many rows in a step take the kernels for long portions
SCRATCH_BYTES = 512 << 20  # of those kernels
BLOCK, WIDE, KEYS = 16, 8, 32  # tokens of a block, blocks of the second kernel's tile, keys of a tile


def lib():
    global _declared
    L = latent.lib()
    if not _declared:
        vp, i32, f32 = ctypes.c_void_p, ctypes.c_int, ctypes.c_float
        head, tail = [vp, vp, i32, f32, vp], [vp] * 6 + [i32] * 12 + [f32, f32]
        L.oxb_joint_simt.argtypes = head + [i32] + tail + [i32, vp]
        L.oxb_joint_decode.argtypes = head + tail + [i32, i32, vp]
        L.oxb_joint_prefill.argtypes = head + tail + [vp, vp, vp, i32, i32, i32, vp, vp, vp, i32, vp]
        L.oxb_joint_decode_supported.argtypes = L.oxb_joint_prefill_supported.argtypes = [i32] * 3
        _declared = True
    return L


def _head(q, kv, layer, out, out_scale):
    return q.data_ptr(), out.data_ptr(), out.stride(0), out_scale, kv.data[layer].data_ptr()


def _tail(q, kv, meta, spec, bias, mix, sink):
    T, H, W = q.shape
    return (meta.block_tables.data_ptr(), meta.seq_lens.data_ptr(), meta.query_start.data_ptr(), _p(sink), _p(mix), _p(bias),
            0 if bias is None else bias.shape[1], meta.seq_lens.shape[0], meta.block_tables.stride(0), T, H, spec.kv_heads, W, ROW_TAIL,
            kv.page_size, kv.num_blocks, spec.window, spec.keep_first, spec.scale, spec.softcap)


def attention_simt(q, kv, layer: int, meta, spec, bias, mix, sink, out, out_scale: float, max_rows: int = _ALL) -> None:
    _check(lib().oxb_joint_simt(*_head(q, kv, layer, out, out_scale), latent.DT[q.dtype], *_tail(q, kv, meta, spec, bias, mix, sink),
                                max_rows, _stream()), "oxb_joint_simt")


def decode_splits(tokens: int, span: int, sms: int, per_sm: int) -> int:
    """CTAs that share a token's keys: ``per_sm`` per SM in all, two pages or more each."""
    return max(1, min(per_sm * sms // max(1, tokens), (span // 16 + 1) // 2, 16 if tokens <= 2 else 8))


def attention_decode(q, kv, layer: int, meta, spec, bias, mix, sink, out, out_scale: float, max_rows: int = _ALL,
                     splits: Optional[int] = None) -> None:
    if splits is None:
        span = meta.max_seq_len or kv.page_size
        if spec.window > 0:
            span = min(span, spec.window + spec.keep_first)
        splits = decode_splits(q.shape[0], span, opcuda.sm_count(q.device), 1 if spec.kv_heads <= 8 else 2)
    _check(lib().oxb_joint_decode(*_head(q, kv, layer, out, out_scale), *_tail(q, kv, meta, spec, bias, mix, sink), max_rows, splits,
                                  _stream()), "oxb_joint_decode")


def most_tiles(lens, window: int, keep_first: int, long_rows: int) -> int:
    """Most tiles of 32 keys that a block of 16 tokens sees."""
    ctx = max(c for n, c in lens if n >= long_rows)
    every = -(-ctx // KEYS)
    return every if window <= 0 else min(every, -(-keep_first // KEYS) + (window + BLOCK - 2) // KEYS + 2)


def blocks_of(lens, long_rows: int):
    """(sequence, first row) of every block of 16 tokens of the long portions, and (first block, blocks) of every group of up to
    eight."""
    seq, row, wide, t = [], [], [], 0
    for b, (n, _) in enumerate(lens):
        if n >= long_rows:
            first = len(seq)
            for r in range(0, n, BLOCK):
                seq.append(b)
                row.append(t + r)
            wide += [(i, min(WIDE, len(seq) - i)) for i in range(first, len(seq), WIDE)]
        t += n
    return seq, row, wide


def _blocks(meta, long_rows: int):
    """:func:`blocks_of` a step on the device, kept for its other layers."""
    key = ("joint_blocks", long_rows)
    got = meta.extra.get(key)
    if got is None:
        seq, row, wide = blocks_of(meta.host_lens, long_rows)
        flat = torch.tensor(seq + row + [v for w in wide for v in w], dtype=torch.int32, device=meta.seq_lens.device)
        n = len(seq)
        got = meta.extra[key] = (flat[:n], flat[n : 2 * n], flat[2 * n :], wide)
    return got


def attention_prefill(q, kv, layer: int, meta, spec, bias, mix, sink, out, out_scale: float, long_rows: int = LONG_ROWS,
                      scratch: int = SCRATCH_BYTES) -> None:
    """Sequences that feed ``long_rows`` rows or more, in launches of as many blocks as the scratch holds."""
    seq, row, wide_dev, wide = _blocks(meta, long_rows)
    H = q.shape[1]
    tiles = most_tiles(meta.host_lens, spec.window, spec.keep_first, long_rows)
    quads = -(-H // 4)
    groups = max(1, scratch // (WIDE * tiles * (quads * 8192 + H * BLOCK * 72)))
    n = min(groups * WIDE, len(seq)) * tiles
    new = lambda size: torch.empty(n * size, dtype=torch.uint8, device=q.device)
    scores, weights, stats = new(quads * 8192), new(H * BLOCK * 64), new(H * BLOCK * 8)
    for w0 in range(0, len(wide), groups):
        part = wide[w0 : w0 + groups]
        b0, b1 = part[0][0], part[-1][0] + part[-1][1]
        _check(lib().oxb_joint_prefill(*_head(q, kv, layer, out, out_scale), *_tail(q, kv, meta, spec, bias, mix, sink), seq.data_ptr(),
                                       row.data_ptr(), wide_dev[2 * w0 :].data_ptr(), b0, b1 - b0, len(part), scores.data_ptr(),
                                       weights.data_ptr(), stats.data_ptr(), tiles, _stream()), "oxb_joint_prefill")


def attention(q, kv, layer: int, meta, spec, bias: Optional[torch.Tensor], mix: Optional[torch.Tensor], sink: Optional[torch.Tensor],
              out: torch.Tensor, out_scale: float) -> None:
    """Attention of a step's queries [T, heads, width] over the cache into ``out`` [T, heads * width] (may be a column slice)."""
    L = lib()
    H, W = q.shape[1:]
    args = (q, kv, layer, meta, spec, bias, mix, sink, out, out_scale)
    fast = q.dtype == torch.bfloat16 and kv.page_size == 16
    short = attention_decode if fast and L.oxb_joint_decode_supported(H, spec.kv_heads, W) else attention_simt
    lens = [n for n, _ in meta.host_lens] if meta.host_lens else [1]
    if not fast or max(lens) < LONG_ROWS or not L.oxb_joint_prefill_supported(H, spec.kv_heads, W):
        short(*args)
        return
    if min(lens) < LONG_ROWS:
        short(*args, LONG_ROWS - 1)
    attention_prefill(*args)
