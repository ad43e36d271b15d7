"""Bindings of the RWKV time-mixing kernels (``csrc/oxb_wkv.cu``), in bfloat16 and float32.  CUDA tensors only; see
:func:`oxidize_b200.ops.wkv_mixer` for the operator's meaning."""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from ..models.config import pad_to
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
        L.oxb_token_shift.argtypes = [vp] * 6 + [i32, vp] + [i32] * 6 + [vp]
        L.oxb_wkv_decay.argtypes = [vp] * 4 + [i32] * 4 + [vp]
        L.oxb_wkv.argtypes = [vp, i32, i32] + [vp] * 7 + [i32, vp] + [i32] * 5 + [f32] + [i32] * 4 + [vp, vp]
        L.oxb_wkv_chunk_bytes.argtypes = [i32]
        _declared = True
    return L


def token_shift(x: torch.Tensor, mu: torch.Tensor, meta, window: torch.Tensor, act_dtype: torch.dtype) -> torch.Tensor:
    """x [T, hidden] float32 to its mixes [n, T, hidden (padded to eight)] with the row ahead (mu [n, hidden]); ``window`` is
    updated."""
    T, H = x.shape
    n, ld = mu.shape[0], pad_to(H, 8)
    out = torch.empty(n, T, ld, dtype=act_dtype, device=x.device)
    _check(lib().oxb_token_shift(x.data_ptr(), mu.data_ptr(), meta.query_start.data_ptr(), meta.seq_lens.data_ptr(),
                                 meta.state_slots.data_ptr(), window.data_ptr(), window.shape[0], out.data_ptr(), latent.DT[act_dtype],
                                 meta.seq_lens.shape[0], T, H, n, ld, _stream()), "oxb_token_shift")
    return out


def log_decay(low: torch.Tensor, w) -> torch.Tensor:
    """[T, heads * width] float32 from the first of the decay's two projections."""
    T, rank = low.shape
    N = w.decay_up.shape[0]
    out = torch.empty(T, N, dtype=torch.float32, device=low.device)
    _check(lib().oxb_wkv_decay(low.data_ptr(), w.decay_up.data_ptr(), w.decay_base.data_ptr(), out.data_ptr(), latent.DT[low.dtype], T, N,
                               rank, _stream()), "oxb_wkv_decay")
    return out


def round_chunks(chunks: int, bytes_per_chunk: int) -> int:
    """Chunks of a round: as many as the scratch limit lets through, in rounds of equal length."""
    rounds = -(-chunks * bytes_per_chunk // SCRATCH_BYTES)
    return max(1, -(-chunks // rounds))


def wkv(z: torch.Tensor, decay: torch.Tensor, w, spec, meta, state: torch.Tensor, eps: float, out: torch.Tensor,
        chunk_rows: Optional[int] = None, rounds: Optional[int] = None) -> None:
    """z [T, r | k | v | gate] to the normed, gated heads ``out`` [T, heads * width]; ``state`` [slots, H, K, K] is updated."""
    H, K, _ = spec.state_shape
    B = meta.seq_lens.shape[0]
    most = max(1, meta.max_query_len)

    def run(lo: int, hi: int, rnd: int = 0, ws: Optional[torch.Tensor] = None) -> None:
        _check(lib().oxb_wkv(z.data_ptr(), z.stride(0), latent.DT[z.dtype], decay.data_ptr(), meta.query_start.data_ptr(),
                             meta.seq_lens.data_ptr(), meta.state_slots.data_ptr(), w.bonus.data_ptr(), w.norm.data_ptr(), state.data_ptr(),
                             state.shape[0], out.data_ptr(), out.stride(0), B, H, K, spec.dim, eps, lo, hi, most, rnd, _p(ws), _stream()),
               "oxb_wkv")

    cut = CHUNK_ROWS if chunk_rows is None else chunk_rows
    size = lib().oxb_wkv_chunk_bytes(K) if z.dtype == torch.bfloat16 and most >= cut else 0
    if size == 0:
        run(1, _ALL)
        return
    if meta.host_lens is None or min(n for n, _ in meta.host_lens) < cut:
        run(1, cut - 1)
    rnd = round_chunks((most + CHUNK - 1) // CHUNK, B * H * size) if rounds is None else rounds
    run(cut, _ALL, rnd, torch.empty(B * rnd * H * size, dtype=torch.uint8, device=z.device))


def wkv_mixer(x: torch.Tensor, w, spec, meta, state: torch.Tensor, window: torch.Tensor, eps: float, act_dtype: torch.dtype) -> torch.Tensor:
    from . import linear

    if meta.state_slots is None:
        raise ValueError("a layer with a recurrent state needs the sequences' state slots")
    T, n = x.shape[0], spec.out_dim
    mixes = token_shift(x, w.mu, meta, window, act_dtype)
    z = torch.empty(T, 4 * n, dtype=act_dtype, device=x.device)
    latent.batched(mixes[:4], w.proj, z, n, 4 * n)
    decay = log_decay(linear(mixes[4], w.decay_down), w)
    out = torch.empty(T, n, dtype=act_dtype, device=x.device)
    wkv(z, decay, w, spec, meta, state, eps, out)
    return out
