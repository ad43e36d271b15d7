"""Bindings of the attention kernels that work on the scores of all heads together (``csrc/oxb_joint.cu``), in bfloat16 and
float32.  CUDA tensors only; see :func:`oxidize_b200.ops.ref.joint_attention` for the operator's meaning."""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from ..models.config import ROW_TAIL
from . import cuda_latent as latent
from .cuda import _check, _p, _stream

_declared = False


def lib():
    global _declared
    L = latent.lib()
    if not _declared:
        vp, i32, f32 = ctypes.c_void_p, ctypes.c_int, ctypes.c_float
        L.oxb_joint_simt.argtypes = [vp, vp, i32, f32, vp, i32] + [vp] * 6 + [i32] * 12 + [f32, f32, vp]
        _declared = True
    return L


def _shape(q, kv, meta, spec, bias):
    T, H, W = q.shape
    return ([0 if bias is None else bias.shape[1], meta.seq_lens.shape[0], meta.block_tables.stride(0), T, H, spec.kv_heads, W, ROW_TAIL,
             kv.page_size, kv.num_blocks, spec.window, spec.keep_first])


def attention_simt(q, kv, layer: int, meta, spec, bias, mix, sink, out, out_scale: float) -> None:
    _check(lib().oxb_joint_simt(q.data_ptr(), out.data_ptr(), out.stride(0), out_scale, kv.data[layer].data_ptr(), latent.DT[q.dtype],
                                meta.block_tables.data_ptr(), meta.seq_lens.data_ptr(), meta.query_start.data_ptr(), _p(sink), _p(mix),
                                _p(bias), *_shape(q, kv, meta, spec, bias), spec.scale, spec.softcap, _stream()), "oxb_joint_simt")


def attention(q, kv, layer: int, meta, spec, bias: Optional[torch.Tensor], mix: Optional[torch.Tensor], sink: Optional[torch.Tensor],
              out: torch.Tensor, out_scale: float) -> None:
    """Attention of a step's queries [T, heads, width] over the cache into ``out`` [T, heads * width] (may be a column slice)."""
    attention_simt(q, kv, layer, meta, spec, bias, mix, sink, out, out_scale)
