"""Bindings of the gated-delta-rule kernels (``csrc/oxb_delta.cu``), in bfloat16 and float32.  CUDA tensors only; see
:func:`oxidize_b200.ops.ref.delta_rule` for the operator's meaning."""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from . import cuda as opcuda
from . import cuda_latent as latent
from .cuda import _check, _p, _stream

_declared = False
_ALL = 1 << 30
SCRATCH_BYTES = 512 << 20  # of the chunk kernels
CHUNK, CHUNK_ROWS = 64, 9  # tokens per chunk; sequences that feed at least CHUNK_ROWS rows in a step go through chunks


def lib():
    global _declared
    L = latent.lib()
    if not _declared:
        vp, i32, f32 = ctypes.c_void_p, ctypes.c_int, ctypes.c_float
        L.oxb_delta.argtypes = ([vp] + [i32] * 5 + [vp] * 4 + [i32, vp, vp, vp, i32, vp, i32, vp, vp, vp, i32, vp, i32, f32]
                                + [i32] * 6 + [f32, f32, i32, i32, i32, i32, i32, i32, vp, vp])
        L.oxb_delta_chunk_bytes.argtypes = [i32, i32]
        L.oxb_delta_window.argtypes = [vp, i32, i32, vp, vp, vp, i32, vp] + [i32] * 6 + [vp]
        _declared = True
    return L


def chunk_values(V: int, heads: int, sms: int) -> int:
    """Values of a head's state per CTA of the kernel that goes from chunk to chunk: the fewer, the shorter each of its steps,
    as long as all CTAs run at once."""
    return 32 if V % 32 == 0 and heads * (V // 16) > sms else 16


def round_chunks(chunks: int, bytes_per_chunk: int) -> int:
    """Chunks of a round: as many as the scratch limit lets through, in rounds of equal length."""
    rounds = -(-chunks * bytes_per_chunk // SCRATCH_BYTES)
    return max(1, -(-chunks // rounds))


def delta_rule(z: torch.Tensor, w, spec, meta, state: torch.Tensor, window: torch.Tensor, eps: float, out: torch.Tensor,
               out_scale: float = 1.0, chunk_rows: Optional[int] = None, values: Optional[int] = None,
               rounds: Optional[int] = None) -> None:
    """z [T, q | k | v | gate | decay | beta] to the normed, gated heads ``out`` [T, heads * v_width] (either may be a column
    slice); ``state`` [slots, H, K, V] and ``window`` [slots, conv, channels] are updated."""
    L = lib()
    H, K, V = spec.state_shape
    G, B, C = spec.kv_heads, meta.seq_lens.shape[0], spec.channels
    if meta.state_slots is None:
        raise ValueError("a layer with a recurrent state needs the sequences' state slots")
    most = max(1, meta.max_query_len)
    dt = latent.DT[z.dtype]

    def run(lo: int, hi: int, nv: int = 0, rnd: int = 1, ws: Optional[torch.Tensor] = None) -> None:
        _check(L.oxb_delta(z.data_ptr(), z.stride(0), dt, C, C + spec.gate_dim, C + spec.gate_dim + spec.decay_dim,
                           meta.query_start.data_ptr(), meta.seq_lens.data_ptr(), meta.state_slots.data_ptr(), w.conv.data_ptr(), spec.conv,
                           w.a_log.data_ptr(), w.dt_bias.data_ptr(), _p(w.decay_up), spec.decay_dim, _p(w.gate_up), spec.gate_dim,
                           w.norm.data_ptr(), state.data_ptr(), window.data_ptr(), state.shape[0], out.data_ptr(), out.stride(0), out_scale,
                           B, H, G, K, V, spec.v_dim, spec.dim ** -0.5, eps, lo, hi, 1 if most == 1 else 0, nv, most, rnd, _p(ws), _stream()),
               "oxb_delta")

    cut = CHUNK_ROWS if chunk_rows is None else chunk_rows
    size = L.oxb_delta_chunk_bytes(K, V) if z.dtype == torch.bfloat16 and most >= cut else 0
    if size == 0:
        low = None
        if most == 1 and z.dtype == torch.bfloat16 and z.shape[0] == B and (w.decay_up is not None or w.gate_up is not None):
            low = torch.empty(B * H * (K + V), dtype=torch.float32, device=z.device)
        run(1, _ALL, ws=low)
    else:
        lens = [n for n, _ in meta.host_lens] if meta.host_lens else [1, most] * B
        if min(lens) < cut:
            run(1, cut - 1)
        long, sms = H * sum(n >= cut for n in lens), opcuda.sm_count(z.device)
        rnd = round_chunks((most + CHUNK - 1) // CHUNK, B * H * size) if rounds is None else rounds
        ws = torch.empty(B * rnd * H * size, dtype=torch.uint8, device=z.device)
        run(cut, _ALL, chunk_values(V, long, sms) if values is None else values, rnd, ws)
    if most > 1:
        _check(L.oxb_delta_window(z.data_ptr(), z.stride(0), dt, meta.query_start.data_ptr(), meta.seq_lens.data_ptr(),
                                  meta.state_slots.data_ptr(), spec.conv, window.data_ptr(), state.shape[0], B, H, G, K, V, _stream()),
               "oxb_delta_window")
