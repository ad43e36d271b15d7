"""One entry for every checkpoint format: configuration, compute type and weights of whatever ``open_checkpoint`` returned."""
from __future__ import annotations

from typing import Optional, Tuple

import torch

from ..formats.layered import Checkpoint, LayeredCheckpoint
from .config import ModelConfig, config_from_gguf
from .layered import config_from_layered, load_layered_weights
from .weights import ModelWeights, load_weights


def config_from_checkpoint(ck: Checkpoint) -> ModelConfig:
    return config_from_layered(ck) if isinstance(ck, LayeredCheckpoint) else config_from_gguf(ck)


def act_dtype_for(cfg: ModelConfig, device: torch.device, compute_dtype: str = "auto") -> torch.dtype:
    """Activation type of a model on a device.  The GPU kernels work in bfloat16; the ones that models with listed layers
    use also exist in float32."""
    if compute_dtype not in ("auto", "bf16", "f32"):
        raise ValueError("compute_dtype must be auto, bf16 or f32")
    if device.type != "cuda":
        return torch.float32
    if compute_dtype == "f32":
        if not cfg.is_layered:
            raise ValueError(f"architecture {cfg.arch!r} has no float32 device kernels (compute_dtype='f32')")
        return torch.float32
    return torch.bfloat16


def load_checkpoint_weights(ck: Checkpoint, cfg: ModelConfig, device="cpu", act_dtype: torch.dtype = torch.float32,
                            tp_rank: int = 0, tp_size: int = 1, ep_rank: int = 0, ep_size: int = 1,
                            layer_range: Optional[Tuple[int, int]] = None, resident_layers: int = 0,
                            transcode: str = "") -> ModelWeights:
    if not isinstance(ck, LayeredCheckpoint):
        return load_weights(ck, cfg, device, act_dtype, tp_rank, tp_size, ep_rank, ep_size, layer_range=layer_range,
                            resident_layers=resident_layers, transcode=transcode)
    if layer_range is not None:
        raise ValueError("a model with per-layer geometry runs as one pipeline stage (layers may share cached rows)")
    if transcode:
        raise ValueError("weights of a layer-list checkpoint are served as stored (no load-time re-encoding)")
    return load_layered_weights(ck, cfg, device, act_dtype, tp_rank, tp_size, resident_layers)
