"""Plain-PyTorch fp32 statement of every operator: the CPU execution path and the oracle
that each sm_100a kernel is tested against.

Semantics follow the reference's CPU kernels: RMSNorm ``y = x * rsqrt(mean(x^2)+eps) * w``
(``compute/tensor/kernels/activation.rs:357``), NeoX split-half *partial* RoPE on the first
``rope_dim`` channels of each head (``activation.rs:98-198``; YaRN scaling included), online
softmax GQA attention (``compute/flash_attention.rs:596,745``), SwiGLU, and the symmetric
per-32-channel KV quantizers (``compute/kv_cache/storage.rs:90-138``).
"""
from __future__ import annotations

import math
from typing import Optional, Tuple

import torch

from ..quant import ref as qref

KV_QBLOCK = 32  # channels per KV quantization block


# --------------------------------------------------------------------------- weights


def dequantize_weight(w) -> torch.Tensor:
    """QTensor -> dense float32 [out, in] (host decode through the NumPy oracle)."""
    if w.qtype in ("F32", "F16", "BF16"):
        return w.data.float()
    if w.qtype == "FP8B":
        codes = w.data.cpu().numpy().reshape(-1)
        scales = w.scales.float().cpu().numpy().reshape(-1)
        out = qref.dequantize_fp8_block(codes, scales, w.block)
        return torch.from_numpy(out).reshape(w.shape).to(w.data.device)
    raw = w.data.cpu().numpy()
    n = w.shape[0] * w.shape[1]
    return torch.from_numpy(qref.dequantize(w.qtype, raw, n).copy()).reshape(w.shape).to(w.data.device)


def linear(x: torch.Tensor, w, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    dense = w.dense_cache()
    y = x.float() @ dense.t()
    if bias is not None:
        y = y + bias.float()
    return y.to(x.dtype)


def embed(tokens: torch.Tensor, table, scale: float = 1.0) -> torch.Tensor:
    dense = table.dense_cache()
    out = dense[tokens.long()]
    return out * scale if scale != 1.0 else out


# --------------------------------------------------------------------------- norms / act


def rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    xf = x.float()
    y = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * w.float()
    return y.to(x.dtype)


def add_rmsnorm(x: torch.Tensor, residual: Optional[torch.Tensor], w: torch.Tensor, eps: float):
    """(normed, new_residual) with new_residual = x + residual (residual kept in x.dtype)."""
    if residual is not None:
        x = (x.float() + residual.float()).to(x.dtype)
    return rmsnorm(x, w, eps), x


def silu_mul(gate_up: torch.Tensor) -> torch.Tensor:
    g, u = gate_up.float().chunk(2, dim=-1)
    return (torch.nn.functional.silu(g) * u).to(gate_up.dtype)


def gelu_mul(gate_up: torch.Tensor) -> torch.Tensor:
    g, u = gate_up.float().chunk(2, dim=-1)
    return (torch.nn.functional.gelu(g, approximate="tanh") * u).to(gate_up.dtype)


def residual_norm(res: Optional[torch.Tensor], y: Optional[torch.Tensor], alpha: float, w: torch.Tensor,
                  b: Optional[torch.Tensor], eps: float, kind: str = "layer", act_dtype: torch.dtype = torch.float32):
    """Norm after the sum: norm(alpha * res + y) in float32, as (float32 stream, the same in ``act_dtype``).  ``layer``
    subtracts the mean and divides by the root of the mean squared deviation; ``rms`` divides by the root mean square."""
    z = y.float() if res is None else (alpha * res.float() if y is None else alpha * res.float() + y.float())
    if kind == "layer":
        z = z - z.mean(-1, keepdim=True)
    z = z * torch.rsqrt(z.pow(2).mean(-1, keepdim=True) + eps) * w.float()
    if b is not None:
        z = z + b.float()
    return z, z.to(act_dtype)


def branch_norm(res: torch.Tensor, y: Optional[torch.Tensor], w_post: Optional[torch.Tensor], w_next: Optional[torch.Tensor],
                eps: float, act_dtype: torch.dtype = torch.float32):
    """Norms on both sides of a branch: x = res + rmsnorm(y) * w_post in float32 and the next branch's input
    rmsnorm(x) * w_next in ``act_dtype``; (x, None) without ``w_next``."""
    x = res.float() if y is None else res.float() + rmsnorm(y.float(), w_post, eps)
    return x, None if w_next is None else rmsnorm(x, w_next, eps).to(act_dtype)


def joint_norm(res: torch.Tensor, mix, ffn, w_next: Optional[torch.Tensor], eps: float, act_dtype: torch.dtype = torch.float32):
    """Both branches of a layer join the stream: x = res + mix + ffn in float32 and the next layer's input rmsnorm(x) * w_next
    in ``act_dtype``; (x, None) without ``w_next``.  ``mix`` may be a pair of outputs with norms and scales of their own."""
    x = res.float()
    if mix is not None:
        y = mix
        if not isinstance(mix, torch.Tensor):
            y = (mix.left_scale * rmsnorm(mix.left.float(), mix.left_norm, eps)
                 + mix.right_scale * rmsnorm(mix.right.float(), mix.right_norm, eps))
        x = x + y.float()
    if ffn is not None:
        x = x + ffn.float()
    return x, None if w_next is None else rmsnorm(x, w_next, eps).to(act_dtype)


def activation(x: torch.Tensor, act: str) -> torch.Tensor:
    """Elementwise activation of a feed-forward block without a gate: ``relu2`` is the square of relu."""
    if act == "relu2":
        return torch.relu(x.float()).square().to(x.dtype)
    raise ValueError(f"unknown activation {act!r}")


# --------------------------------------------------------------------------- rope


def rope_inv_freq(rotary_dim: int, theta: float, scaling=None, device=None, freq_factors=None,
                  dtype: torch.dtype = torch.float32) -> torch.Tensor:
    """Per-pair inverse frequencies [rotary_dim/2] with optional linear / YaRN scaling.  ``freq_factors``
    ([rotary_dim/2], from a ``rope_freqs.weight`` / ``rope_factors_*.weight`` tensor of the checkpoint) divides each
    frequency: that is how Llama-3.1-style and LongRoPE context extensions are stored in GGUF files."""
    half = rotary_dim // 2
    idx = torch.arange(half, dtype=torch.float64, device=device)
    inv = theta ** (-2.0 * idx / rotary_dim)
    if scaling is not None and scaling.type == "linear" and scaling.factor > 0:
        inv = inv / scaling.factor
    elif (scaling is not None and scaling.type == "yarn" and scaling.original_context_length > 0
          and (scaling.factor > 1 or scaling.magnitude > 0)):
        orig = scaling.original_context_length

        def corr_dim(n_rot):
            return rotary_dim * math.log(orig / (n_rot * 2 * math.pi)) / (2 * math.log(theta))

        lo = max(math.floor(corr_dim(scaling.beta_fast)), 0)
        hi = min(math.ceil(corr_dim(scaling.beta_slow)), scaling.ramp_limit or half - 1)
        ramp = ((idx - lo) / max(hi - lo, 1e-3)).clamp(0, 1)
        mix = 1.0 - ramp  # 1 => extrapolate (keep), 0 => interpolate
        inv = inv / scaling.factor * (1 - mix) + inv * mix
    if freq_factors is not None:
        ff = torch.as_tensor(freq_factors, dtype=torch.float64, device=inv.device).reshape(-1)
        if ff.numel() < half:
            raise ValueError(f"rope frequency factors have {ff.numel()} entries, the rotary half dimension is {half}")
        inv = inv / ff[:half]
    return inv.to(dtype)


def rope_mscale(scaling) -> float:
    if scaling is not None and scaling.magnitude > 0:
        return scaling.magnitude
    if scaling is not None and scaling.type == "yarn" and scaling.factor > 1:
        return 0.1 * math.log(scaling.factor) + 1.0
    return 1.0


def apply_rope(x: torch.Tensor, positions: torch.Tensor, inv_freq: torch.Tensor, pairing: str = "split_half",
               mscale: float = 1.0) -> torch.Tensor:
    """x: [T, n_heads, head_dim]; rotates the first 2*len(inv_freq) channels of each head."""
    half = inv_freq.numel()
    rot = 2 * half
    ang = positions.double()[:, None] * inv_freq.double()[None, :]
    cos = (ang.cos() * mscale).float()[:, None, :]
    sin = (ang.sin() * mscale).float()[:, None, :]
    xf = x.float()
    xr = xf[..., :rot]
    if pairing == "split_half":
        a, b = xr[..., :half], xr[..., half:]
        out = torch.cat([a * cos - b * sin, b * cos + a * sin], dim=-1)
    else:
        a, b = xr[..., 0::2], xr[..., 1::2]
        out = torch.stack([a * cos - b * sin, b * cos + a * sin], dim=-1).flatten(-2)
    return torch.cat([out, xf[..., rot:]], dim=-1).to(x.dtype)


# --------------------------------------------------------------------------- KV cache


def kv_quantize(x: torch.Tensor, bits: int):
    """Symmetric per-32-channel quantization: returns (codes uint8, scales f32).

    q8: code = q + 127 with q in [-127,127]; q4: code = q + 7 with q in [-7,7], two codes per
    byte, low nibble first (storage.rs:90-138)."""
    xf = x.float().reshape(*x.shape[:-1], -1, KV_QBLOCK)
    qmax = 127.0 if bits == 8 else 7.0
    amax = xf.abs().amax(-1, keepdim=True)
    scale = amax / qmax
    inv = torch.where(scale > 0, 1.0 / scale, torch.zeros_like(scale))
    q = torch.round(xf * inv).clamp(-qmax, qmax) + qmax
    q = q.to(torch.uint8).reshape(*x.shape)
    if bits == 4:
        q = q[..., 0::2] | (q[..., 1::2] << 4)
    return q, scale.squeeze(-1)


def kv_dequantize(codes: torch.Tensor, scales: torch.Tensor, bits: int) -> torch.Tensor:
    if bits == 4:
        lo = (codes & 0xF).float() - 7.0
        hi = (codes >> 4).float() - 7.0
        q = torch.stack([lo, hi], dim=-1).flatten(-2)
    else:
        q = codes.float() - 127.0
    q = q.reshape(*q.shape[:-1], -1, KV_QBLOCK) * scales.unsqueeze(-1)
    return q.flatten(-2)


def kv_write(kv, layer: int, k: torch.Tensor, v: Optional[torch.Tensor], slot_mapping: torch.Tensor) -> None:
    """Scatter post-RoPE K/V rows [T, n_kv, hd] into the paged cache at flat slots (``v`` None: a cache of single rows)."""
    page = kv.page_size
    slots = slot_mapping.long()
    valid = slots >= 0
    if not bool(valid.all()):
        k, v, slots = k[valid], None if v is None else v[valid], slots[valid]
    blk, off = slots // page, slots % page
    data = kv.data[layer]
    if kv.dtype_name in ("f16", "bf16", "f32"):
        data[blk, :, 0, off] = k.to(data.dtype)
        if v is not None:
            data[blk, :, 1, off] = v.to(data.dtype)
    else:
        bits = 8 if kv.dtype_name == "q8" else 4
        kc, ks = kv_quantize(k, bits)
        data[blk, :, 0, off] = kc
        kv.scales[layer][blk, :, 0, off] = ks
        if v is not None:
            vc, vs = kv_quantize(v, bits)
            data[blk, :, 1, off] = vc
            kv.scales[layer][blk, :, 1, off] = vs


def kv_gather(kv, layer: int, block_table: torch.Tensor, seq_len: int) -> Tuple[torch.Tensor, torch.Tensor]:
    """Dense (K, V) [seq_len, n_kv, hd] float32 of one sequence, through its block table."""
    page = kv.page_size
    nb = (seq_len + page - 1) // page
    blocks = block_table[:nb].long()
    d = kv.data[layer][blocks]  # [nb, n_kv, 2, page, hd or packed]
    if kv.dtype_name in ("q8", "q4"):
        bits = 8 if kv.dtype_name == "q8" else 4
        d = kv_dequantize(d, kv.scales[layer][blocks], bits)
    d = d.float().permute(2, 0, 3, 1, 4).reshape(2, nb * page, d.shape[1], -1)[:, :seq_len]
    return d[0], d[1]


def paged_attention(q: torch.Tensor, kv, layer: int, meta, scale: float, sliding_window: int = 0,
                    softcap: float = 0.0, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal GQA attention of packed query rows against the paged cache.

    q: [T, n_heads, hd].  For sequence b the rows ``query_start[b]:query_start[b+1]`` are its
    last ``qlen`` positions (context length ``seq_lens[b]`` already includes them), so one
    code path covers decode (qlen 1), chunked prefill and speculative verify (qlen K+1).
    ``softcap`` > 0 replaces the scaled scores by ``softcap * tanh(scores / softcap)`` before masking (Gemma-2);
    ``sink`` [heads] is a logit that joins the softmax denominator only."""
    T, nh, hd = q.shape
    out = torch.zeros(T, nh, hd, dtype=torch.float32, device=q.device)
    qs = meta.query_start.tolist()
    sl = meta.seq_lens.tolist()
    for b in range(len(sl)):
        t0, t1 = qs[b], qs[b + 1]
        qlen = t1 - t0
        if qlen == 0:
            continue
        L = sl[b]
        K, V = kv_gather(kv, layer, meta.block_tables[b], L)
        nkv = K.shape[1]
        g = nh // nkv
        qb = q[t0:t1].float().reshape(qlen, nkv, g, hd)
        s = torch.einsum("qkgd,lkd->kgql", qb, K) * scale
        if softcap > 0:
            s = torch.tanh(s / softcap) * softcap
        qpos = torch.arange(L - qlen, L, device=q.device)[:, None]
        kpos = torch.arange(L, device=q.device)[None, :]
        mask = kpos <= qpos
        if sliding_window > 0:
            mask &= kpos > qpos - sliding_window
        s = s.masked_fill(~mask, float("-inf"))
        p = softmax_sink(s, None if sink is None else sink.reshape(nkv, g, 1, 1))
        o = torch.einsum("kgql,lkd->qkgd", p, V)
        out[t0:t1] = o.reshape(qlen, nh, hd)
    return out.to(q.dtype)


def latent_rows(qkv: torch.Tensor, m, spec, rope, meta, kv, layer: int, eps: float) -> torch.Tensor:
    """From the projections of a latent-attention layer ([queries | latent | rotary key], the last two only where the
    layer owns cache rows) write this step's cache rows and return the queries in absorbed form [T, H, row_dim]: the
    position-free part multiplied by W_uk, the rotated part behind it, zeros in the padding."""
    H, nope, rot, c = m.w_uk.shape[0], spec.nope_dim, spec.rope_dim, spec.kv_rank
    T, pad, width = qkv.shape[0], spec.latent_pad, spec.row_dim
    q = qkv[:, : H * spec.qk_dim].reshape(T, H, spec.qk_dim)
    if spec.kv_from is None:
        ckv = qkv[:, H * spec.qk_dim :]
        row = torch.zeros(T, 1, width, dtype=qkv.dtype, device=qkv.device)
        row[:, 0, :c] = rmsnorm(ckv[:, :c], m.kv_a_norm, eps)
        row[:, :, pad : pad + rot] = apply_rope(ckv[:, None, c:], meta.positions, rope.inv_freq, rope.pairing, rope.mscale)
        kv_write(kv, layer, row, None, meta.slot_mapping)
    out = torch.zeros(T, H, width, dtype=qkv.dtype, device=qkv.device)
    out[:, :, :c] = torch.einsum("thn,hnc->thc", q[:, :, :nope].float(), m.w_uk.float())
    out[:, :, pad : pad + rot] = apply_rope(q[:, :, nope:], meta.positions, rope.inv_freq, rope.pairing, rope.mscale)
    return out


def softmax_sink(s: torch.Tensor, sink: Optional[torch.Tensor]) -> torch.Tensor:
    """Softmax over the last axis; ``sink`` (a logit per row, broadcast against ``s[..., :1]``) joins the denominator only."""
    if sink is None:
        return torch.softmax(s, dim=-1)
    sk = sink.float().expand(*s.shape[:-1], 1)
    return torch.softmax(torch.cat([s, sk], dim=-1), dim=-1)[..., :-1]


def latent_attention(q: torch.Tensor, kv, layer: int, meta, scale: float, latent_dim: int, window: int = 0,
                     sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Multi-query attention over latent cache rows (DeepSeek latent attention in absorbed form).

    q: [T, H, latent_dim + rope]; the cache holds one row of that width per token, shared by all heads, and the value of
    a row is its first ``latent_dim`` entries.  ``window`` > 0 keeps the latest ``window`` positions of each query (itself
    included); ``sink`` [H] is a logit that joins the softmax denominator only.  Returns [T, H, latent_dim].  A decode step (one row per sequence) is one
    batched gather + two batched matrix products over all sequences; other steps go sequence by sequence.  Device-agnostic
    torch: this is what runs on a GPU too, where the attention kernel has no 576-wide head."""
    T, H, D = q.shape
    B = int(meta.seq_lens.shape[0])
    page = kv.page_size
    quant = kv.dtype_name in ("q8", "q4")

    def rows_of(blocks: torch.Tensor) -> torch.Tensor:  # [..., nb] block ids -> [..., nb * page, D] float32 key rows
        d = kv.data[layer][blocks]  # [..., nb, 1, 2, page, D or packed]
        if quant:
            d = kv_dequantize(d, kv.scales[layer][blocks], 8 if kv.dtype_name == "q8" else 4)
        d = d[..., 0, 0, :, :].float()
        return d.reshape(*d.shape[:-3], d.shape[-3] * page, d.shape[-1])

    if T == B and meta.max_query_len == 1:
        max_len = int(meta.max_seq_len) or int(meta.seq_lens.max())
        nb = (max_len + page - 1) // page
        K = rows_of(meta.block_tables[:, :nb].long())[:, :max_len]  # [B, L, D]
        s = torch.einsum("bhd,bld->bhl", q.float(), K) * scale
        kpos = torch.arange(max_len, device=q.device)[None, :]
        live = kpos < meta.seq_lens.long()[:, None]
        if window > 0:
            live &= kpos >= meta.seq_lens.long()[:, None] - window
        s = s.masked_fill(~live[:, None, :], float("-inf"))
        p = softmax_sink(s, None if sink is None else sink[None, :, None])
        return torch.einsum("bhl,blc->bhc", p, K[..., :latent_dim]).to(q.dtype)
    out = torch.zeros(T, H, latent_dim, dtype=torch.float32, device=q.device)
    qs, sl = meta.query_start.tolist(), meta.seq_lens.tolist()
    for b in range(B):
        t0, t1 = qs[b], qs[b + 1]
        n, L = t1 - t0, sl[b]
        if n == 0:
            continue
        K = rows_of(meta.block_tables[b, : (L + page - 1) // page].long())[:L]  # [L, D]
        s = torch.einsum("qhd,ld->hql", q[t0:t1].float(), K) * scale
        kpos, qpos = torch.arange(L, device=q.device)[None, :], torch.arange(L - n, L, device=q.device)[:, None]
        seen = kpos <= qpos
        if window > 0:
            seen &= kpos > qpos - window
        s = s.masked_fill(~seen[None], float("-inf"))
        p = softmax_sink(s, None if sink is None else sink[:, None, None])
        out[t0:t1] = torch.einsum("hql,lc->qhc", p, K[:, :latent_dim])
    return out.to(q.dtype)


# --------------------------------------------------------------------------- listed mixers


def padded_norm(x: torch.Tensor, w: torch.Tensor, n: int, eps: float) -> torch.Tensor:
    """RMS norm over the last axis of zero-padded rows that hold ``n`` values."""
    return x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / n + eps) * w


def query_temperature(positions: torch.Tensor, coef: float, every: float) -> torch.Tensor:
    return 1.0 + coef * torch.log(torch.floor((positions.float() + 1.0) / every) + 1.0)


def head_prep(z: torch.Tensor, q_norm, k_norm, spec, rope, meta, kv, layer: int, eps: float, v_first: Optional[torch.Tensor] = None,
              v_mix: Optional[torch.Tensor] = None) -> torch.Tensor:
    """From a layer's q | k | v projections (heads of ``spec.width`` values): norms, rotation, query temperature, values mixed
    with ``v_first`` [T, kv_heads, v_dim or more], this step's cache rows; the queries [T, heads, width]."""
    T, H, G, W = z.shape[0], spec.heads, spec.kv_heads, spec.width
    q, k, v = z[:, : H * W].float(), z[:, H * W : (H + G) * W].float(), z[:, (H + G) * W : (H + 2 * G) * W]
    if spec.qk_norm == "full":
        q, k = padded_norm(q, q_norm, H * spec.dim, eps), padded_norm(k, k_norm, G * spec.dim, eps)
    q, k = q.reshape(T, H, W), k.reshape(T, G, W)
    if spec.qk_norm == "head":
        q, k = padded_norm(q, q_norm, spec.dim, eps), padded_norm(k, k_norm, spec.dim, eps)
    if rope is not None:
        q = apply_rope(q, meta.positions, rope.inv_freq, rope.pairing, rope.mscale)
        k = apply_rope(k, meta.positions, rope.inv_freq, rope.pairing, rope.mscale)
    if spec.temp_coef != 0.0:
        q = q * query_temperature(meta.positions, spec.temp_coef, spec.temp_every)[:, None, None]
    v = v.reshape(T, G, W)
    if v_first is not None:
        v = v.float().clone()
        v[..., : spec.v_dim] = (1.0 - v_mix) * v[..., : spec.v_dim] + v_mix * v_first[..., : spec.v_dim].float()
    kv_write(kv, layer, k, v, meta.slot_mapping)
    return q.to(z.dtype)


def head_gate(o: torch.Tensor, gate: torch.Tensor, spec) -> torch.Tensor:
    """Heads' outputs [T, heads, width] times the sigmoid of their gates (one per head, or per value)."""
    T = o.shape[0]
    g = torch.sigmoid(gate.float())
    g = g[:, : spec.heads, None] if spec.gate == "head" else g.reshape(T, spec.heads, spec.width)
    return (o.float() * g).to(o.dtype)


def retention(z: torch.Tensor, spec, rope, meta, state: torch.Tensor, eps: float) -> torch.Tensor:
    """Retention of one layer, token by token: z [T, q | k | v | gate], state [slots, heads, k_width, v_width] (updated);
    a sequence whose rows start at position 0 starts from a zero state.  Returns [T, heads * v_width]."""
    T, H, K, V = z.shape[0], spec.heads, spec.k_width, spec.v_width
    z = z.float()
    q, k = z[:, : H * K].reshape(T, H, K), z[:, H * K : 2 * H * K].reshape(T, H, K)
    v, g = z[:, 2 * H * K : 2 * H * K + H * V].reshape(T, H, V), z[:, 2 * H * K + H * V :].reshape(T, H, V)
    q = apply_rope(q, meta.positions, rope.inv_freq, rope.pairing, rope.mscale)
    k = apply_rope(k, meta.positions, rope.inv_freq, rope.pairing, rope.mscale) * spec.dim ** -0.5
    decay = torch.tensor(spec.decay, dtype=torch.float32, device=z.device)[:, None, None]
    o = torch.zeros(T, H, V, dtype=torch.float32, device=z.device)
    qs, lens, slots = meta.query_start.tolist(), meta.seq_lens.tolist(), meta.state_slots.tolist()
    for b in range(len(lens)):
        t0, t1 = qs[b], qs[b + 1]
        if slots[b] < 0 or t1 == t0:
            continue
        S = torch.zeros_like(state[slots[b]]) if lens[b] == t1 - t0 else state[slots[b]]
        for t in range(t0, t1):
            S = decay * S + k[t][:, :, None] * v[t][:, None, :]
            o[t] = (S * q[t][:, :, None]).sum(1)
        state[slots[b]] = S
    y = padded_norm(o, 1.0, spec.v_dim, eps) * torch.nn.functional.silu(g)
    return y.reshape(T, H * V)


def delta_rule(z: torch.Tensor, w, spec, meta, state: torch.Tensor, window: torch.Tensor, eps: float) -> torch.Tensor:
    """Gated delta rule of one layer, token by token: z [T, q | k | v | gate | decay | beta] (``spec``:
    ``models.config.DeltaSpec``), state [slots, heads, k_width, v_width] and the ring of convolution inputs ``window`` [slots,
    conv, channels] (both updated); a sequence whose rows start at position 0 starts from nothing.  [T, heads * v_width]."""
    T, H, G, K, V, n = z.shape[0], spec.heads, spec.kv_heads, spec.k_width, spec.v_width, spec.conv
    F = torch.nn.functional
    C = spec.channels
    zf = z.float()
    u, gate, decay = zf[:, :C], zf[:, C : C + spec.gate_dim], zf[:, C + spec.gate_dim : C + spec.gate_dim + spec.decay_dim]
    beta = torch.sigmoid(zf[:, C + spec.gate_dim + spec.decay_dim :][:, :H])
    gate = torch.sigmoid(gate @ w.gate_up.float().t()) if spec.gate_rank else F.silu(gate)
    a = (decay @ w.decay_up.float().t()) if spec.decay_rank else decay[:, :H]
    g = torch.exp(-torch.exp(w.a_log)[None, :, None] * F.softplus(a + w.dt_bias).reshape(T, H, -1))
    o = torch.zeros(T, H, V, dtype=torch.float32, device=z.device)
    qs, lens, slots = meta.query_start.tolist(), meta.seq_lens.tolist(), meta.state_slots.tolist()
    unit = lambda t: t * torch.rsqrt(t.pow(2).sum(-1, keepdim=True) + 1e-6)
    for b in range(len(lens)):
        t0, t1 = qs[b], qs[b + 1]
        m = t1 - t0
        if slots[b] < 0 or m == 0:
            continue
        pos0, ring = lens[b] - m, window[slots[b]]
        past = torch.stack([ring[p % n] if p >= 0 else torch.zeros_like(ring[0]) for p in range(pos0 - n + 1, pos0)] or [ring[0]])
        rows = torch.cat([past[: n - 1], u[t0:t1]])
        y = F.silu(sum(w.conv[j] * rows[j : j + m] for j in range(n)))
        for p in range(max(pos0, pos0 + m - n), pos0 + m):
            ring[p % n] = u[t0 + p - pos0]
        q = unit(y[:, : G * K].reshape(m, G, K)).repeat_interleave(H // G, dim=1) * spec.dim ** -0.5
        k = unit(y[:, G * K : 2 * G * K].reshape(m, G, K)).repeat_interleave(H // G, dim=1)
        v = y[:, 2 * G * K :].reshape(m, H, V)
        S = torch.zeros_like(state[slots[b]]) if pos0 == 0 else state[slots[b]]
        for t in range(m):
            S = g[t0 + t][:, :, None] * S
            S = S + k[t][:, :, None] * (beta[t0 + t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1)))[:, None, :]
            o[t0 + t] = (S * q[t][:, :, None]).sum(1)
        state[slots[b]] = S
    return padded_norm(o, w.norm, spec.v_dim, eps).reshape(T, H * V) * gate


def grouped_norm(x: torch.Tensor, w: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    parts = x.float().unflatten(-1, (groups, -1))
    return (parts * torch.rsqrt(parts.pow(2).mean(-1, keepdim=True) + eps)).flatten(-2) * w


def add_normed(res: torch.Tensor, y, w: torch.Tensor, groups: int, eps: float, act_dtype, streams=None, depth=None):
    x = res + grouped_norm(y, w, groups, eps)
    if streams is not None:
        streams.results[streams.n] = x
        streams.n += 1
        x = depth[0] * streams.first + torch.einsum("l,lth->th", depth[1:], streams.results[: streams.n])
    return x, None if act_dtype is None else x.to(act_dtype)


def token_shift(x: torch.Tensor, mu: torch.Tensor, meta, window: torch.Tensor) -> torch.Tensor:
    """Mixes of every token's input with the one ahead of it: x [T, hidden] float32, mu [n, hidden] to [n, T, hidden];
    ``window`` [slots, 1, hidden] holds the last input of earlier steps (updated)."""
    before = torch.zeros_like(x)
    qs, lens, slots = meta.query_start.tolist(), meta.seq_lens.tolist(), meta.state_slots.tolist()
    for b in range(len(lens)):
        t0, t1 = qs[b], qs[b + 1]
        if t1 == t0:
            continue
        before[t0 + 1 : t1] = x[t0 : t1 - 1]
        if slots[b] >= 0:
            if lens[b] > t1 - t0:
                before[t0] = window[slots[b], 0]
            window[slots[b], 0] = x[t1 - 1]
    return x + (before - x) * mu[:, None, :]


def wkv_log_decay(low: torch.Tensor, w) -> torch.Tensor:
    """Logarithms of the decays [T, heads * k_width], never positive, from the first of their two projections."""
    return -torch.exp(torch.tanh(low.float()) @ w.decay_up.float().t() + w.decay_base)


def wkv(rkvg: torch.Tensor, log_decay: torch.Tensor, w, spec, meta, state: torch.Tensor, eps: float) -> torch.Tensor:
    """RWKV time mixing of one layer, token by token: rkvg [4, T, heads * width], state [slots, heads, k_width, v_width]
    (updated); a sequence whose rows start at position 0 starts from a zero state.  Returns [T, heads * v_width] float32."""
    T, H, K = rkvg.shape[1], spec.heads, spec.k_width
    r, k, v, g = rkvg.float().unflatten(2, (H, K))
    decay, u = torch.exp(log_decay.float()).unflatten(1, (H, K)), w.bonus.reshape(H, K)
    o = torch.zeros(T, H, K, dtype=torch.float32, device=r.device)
    qs, lens, slots = meta.query_start.tolist(), meta.seq_lens.tolist(), meta.state_slots.tolist()
    for b in range(len(lens)):
        t0, t1 = qs[b], qs[b + 1]
        if slots[b] < 0 or t1 == t0:
            continue
        S = torch.zeros_like(state[slots[b]]) if lens[b] == t1 - t0 else state[slots[b]]
        for t in range(t0, t1):
            o[t] = (S * r[t][:, :, None]).sum(1) + (r[t] * u * k[t]).sum(-1, keepdim=True) * v[t]
            S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        state[slots[b]] = S
    y = padded_norm(o, w.norm.reshape(H, K), spec.dim, eps) * torch.nn.functional.silu(g)
    return y.reshape(T, H * K)


def unit_heads(x: torch.Tensor, n: int, eps: float) -> torch.Tensor:
    """Zero-padded heads that hold ``n`` values over their root mean squares."""
    return padded_norm(x.float(), 1.0, n, eps)


def joint_prep(z: torch.Tensor, spec, meta, kv, layer: int, eps: float) -> torch.Tensor:
    """From a layer's q | k projections (heads of ``spec.width`` values): this step's cache rows, keys as projected with one over
    their root mean square behind them; the queries [T, heads, width] over theirs."""
    T, H, G, W = z.shape[0], spec.heads, spec.kv_heads, spec.width
    q, k = z[:, : H * W].reshape(T, H, W), z[:, H * W : (H + G) * W].reshape(T, G, W)
    row = torch.zeros(T, G, spec.cache_shape[2], dtype=z.dtype, device=z.device)
    row[..., :W] = k
    row[..., W] = torch.rsqrt(k.float().pow(2).sum(-1) / spec.dim + eps)
    kv_write(kv, layer, row, None, meta.slot_mapping)
    return unit_heads(q, spec.dim, eps).to(z.dtype)


def visible(qpos: torch.Tensor, kpos: torch.Tensor, window: int, keep_first: int) -> torch.Tensor:
    """Which keys a query sees: those up to it that are in its window (0: all) or among the first ``keep_first``."""
    seen = kpos <= qpos
    return seen & ((kpos > qpos - window) | (kpos < keep_first)) if window > 0 else seen


def joint_attention(q: torch.Tensor, kv, layer: int, meta, spec, bias: Optional[torch.Tensor], mix: Optional[torch.Tensor],
                    sink: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    """Attention on the scores of all heads together: soft-capped, mixed over the heads by ``mix``, plus ``bias`` [heads,
    distances] (of the mixed scores; the last one serves all further distances).  One cached row is key and value."""
    T, H, W = q.shape
    out = torch.zeros(T, H, W, dtype=torch.float32, device=q.device)
    qs, lens = meta.query_start.tolist(), meta.seq_lens.tolist()
    per = H // spec.kv_heads
    for b in range(len(lens)):
        t0, t1 = qs[b], qs[b + 1]
        n, L = t1 - t0, lens[b]
        if n == 0:
            continue
        nb = (L + kv.page_size - 1) // kv.page_size
        rows = kv.data[layer][meta.block_tables[b][:nb].long()][:, :, 0].float()  # [pages, heads, page, row]
        k = rows.transpose(1, 2).reshape(-1, spec.kv_heads, rows.shape[-1])[:L, :, :W].repeat_interleave(per, dim=1)
        s = torch.einsum("qhd,lhd->hql", q[t0:t1].float(), unit_heads(k, spec.dim, eps)) * spec.scale
        if spec.softcap > 0:
            s = torch.tanh(s / spec.softcap) * spec.softcap
        if mix is not None:
            s = torch.einsum("hg,gql->hql", mix, s)
        qpos, kpos = torch.arange(L - n, L, device=q.device)[:, None], torch.arange(L, device=q.device)[None, :]
        if bias is not None:
            s = s + bias[:, (qpos - kpos).clamp(0, bias.shape[1] - 1)]
        s = s.masked_fill(~visible(qpos, kpos, spec.window, spec.keep_first)[None], float("-inf"))
        p = softmax_sink(s, None if sink is None else sink[:, None, None])
        out[t0:t1] = torch.einsum("hql,lhd->qhd", p, k)
    return out.to(q.dtype)


# --------------------------------------------------------------------------- MoE routing


def moe_route(logits: torch.Tensor, cfg, bias: Optional[torch.Tensor] = None):
    """Router: returns (expert_ids [T,k] int32, weights [T,k] float32).

    softmax → top-k → renormalise (Mixtral/Qwen), or sigmoid(+bias for *selection* only)
    → optional group-limited top-k → unbiased weights → renorm → scale (DeepSeek), as in
    ``moe_ffn_forward_weights`` (model/inference.rs:1690-1804)."""
    lf = logits.float()
    k = cfg.n_experts_used
    if cfg.expert_gating == "sigmoid":
        scores = torch.sigmoid(lf)
    else:
        scores = torch.softmax(lf, dim=-1)
    sel = scores + bias.float() if bias is not None else scores
    if cfg.expert_group_count > 1 and cfg.expert_group_used_count > 0:
        T, E = sel.shape
        gs = E // cfg.expert_group_count
        grp = sel.reshape(T, cfg.expert_group_count, gs)
        if bias is not None:
            gscore = grp.topk(min(2, gs), dim=-1).values.sum(-1)
        else:
            gscore = grp.amax(-1)
        keep = gscore.topk(cfg.expert_group_used_count, dim=-1).indices
        gmask = torch.zeros_like(gscore, dtype=torch.bool).scatter_(1, keep, True)
        sel = sel.masked_fill(~gmask[:, :, None].expand(T, cfg.expert_group_count, gs).reshape(T, E), float("-inf"))
    # stable tie rule: lowest expert index first
    order = torch.sort(sel, dim=-1, descending=True, stable=True).indices[:, :k]
    w = torch.gather(scores, 1, order)
    if cfg.expert_weights_norm:
        w = w / w.sum(-1, keepdim=True).clamp_min(1e-20)
    w = w * cfg.expert_weights_scale
    return order.to(torch.int32), w


# --------------------------------------------------------------------------- sampling


def argmax(logits: torch.Tensor, tie: str = "lowest") -> torch.Tensor:
    """Row argmax; ``tie='highest'`` reproduces the Rust engine's ``max_by`` (last maximal
    element, sampling.rs:236-246), ``'lowest'`` the C port's rule (cuda_fast.cu:506-513)."""
    lf = logits.float()
    if tie == "highest":
        V = lf.shape[-1]
        return (V - 1 - torch.flip(lf, dims=[-1]).argmax(-1)).to(torch.int32)
    return lf.argmax(-1).to(torch.int32)
