"""Throughput of a model that lists its layers (Vefilix: latent attention in a window, norm after the sum) beside the
closest uniform models at equal size, one GPU, random weights:

    python bench.py --layered 4096x32 --steps 32 --warmup 4

Three models of the same width, depth and parameter count per layer are timed: the layered one, a DeepSeek-style latent
attention model (``deepseek2``, same latent geometry, gated feed-forward) and a grouped-query one (``llama``).  Decode: captured
steps replayed, every sequence past its window.  Prefill: portions of 2048 tokens behind 2048 (window 1024) or 4096 tokens.
Then the kernels that differ, each over buffers larger than the L2 in turn, against the measured copy bandwidth."""
from __future__ import annotations

import json
import os

import torch

PAGE, VOCAB, LAYERS = 16, 32000, 8
DIM, ROT, VDIM, RANK = 128, 64, 128, 512


def _peaks():
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "MEASURED_PEAKS.json")
    try:
        with open(path) as f:
            p = json.load(f)
        return float(p["hbm_gbs"]), float(p["bf16_tflops"])
    except (OSError, KeyError, ValueError):
        return 6650.0, 1590.0


def layered(width: int, heads: int, window: int):
    from oxidize_b200.models.config import FeedForwardSpec, LatentAttentionSpec, LayerSpec, RopeScaling, RotarySpec
    from oxidize_b200.models.layered import layered_config

    rot = RotarySpec(ROT, 1e6, RopeScaling("yarn", 4.0, 8192, 32.0, 1.0, ramp_limit=ROT - 1, magnitude=1.1386))
    specs = [LayerSpec(LatentAttentionSpec(heads, DIM, ROT, VDIM, RANK, (DIM + ROT) ** -0.5, rot, window, True,
                                           None if i < LAYERS // 2 else LAYERS // 2 - 1), FeedForwardSpec(4 * width))
             for i in range(LAYERS)]
    return layered_config("vefilix", VOCAB, width, specs, 1e-5, "layer", 2.0, True)


def uniform(kind: str, width: int, heads: int, window: int):
    from oxidize_b200.models.config import ModelConfig

    ffn = (8 * width // 3 + 127) // 128 * 128  # three matrices instead of two
    base = dict(vocab_size=VOCAB, hidden_size=width, n_layers=LAYERS, n_heads=heads, ffn_size=ffn, context_length=1 << 16)
    if kind == "llama":
        return ModelConfig(arch="llama", n_kv_heads=max(1, heads // 4), head_dim=128, sliding_window=window, **base)
    return ModelConfig(arch="deepseek2", n_kv_heads=heads, head_dim=DIM + ROT, rope_dim=ROT, qk_nope_dim=DIM, v_head_dim=VDIM,
                       kv_lora_rank=RANK, rope_pairing="adjacent", **base)


def weights(cfg, dev):
    from oxidize_b200.models.weights import LayerWeights, LinearWeight, MLAWeights, ModelWeights, QTensor
    from oxidize_b200.utils.synth import synth_weights

    if not cfg.is_mla:
        return synth_weights(cfg, dev, "BF16", seed=0)

    def q(o, i):
        return QTensor("BF16", (torch.randn(o, i, device=dev) * 0.02).bfloat16(), (o, i))

    one = lambda n: torch.ones(n, device=dev)
    h, H = cfg.hidden_size, cfg.n_heads
    layers = [LayerWeights(attn_norm=one(h), wqkv=None, wo=LinearWeight([q(h, H * VDIM)]), ffn_norm=one(h),
                           mla=MLAWeights(q(RANK + ROT, h), one(RANK), q(H * DIM, RANK).data.reshape(H, DIM, RANK),
                                          q(H * VDIM, RANK).data.reshape(H, VDIM, RANK), q=LinearWeight([q(H * (DIM + ROT), h)])),
                           w_gate_up=LinearWeight([q(2 * cfg.ffn_size, h)]), w_down=LinearWeight([q(h, cfg.ffn_size)]))
              for _ in range(cfg.n_layers)]
    return ModelWeights(cfg, q(cfg.vocab_size, h), layers, one(h), LinearWeight([q(cfg.vocab_size, h)]))


def timed(fn, steps: int, warmup: int) -> float:
    """Milliseconds per call, CUDA events around ``steps`` calls."""
    for _ in range(max(3, warmup)):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(steps):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / steps


def captured(fn):
    s = torch.cuda.Stream()
    s.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(s):
        for _ in range(2):
            fn()
    torch.cuda.current_stream().wait_stream(s)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        fn()
    return g


def batch(B: int, rows: int, ctx: int, dev):
    from oxidize_b200.models.transformer import BatchMeta

    nb = (ctx + PAGE - 1) // PAGE
    i32 = dict(dtype=torch.int32, device=dev)
    bt = torch.randperm(B * nb, device=dev).reshape(B, nb).int()
    pos = torch.arange(ctx - rows, ctx, **i32).repeat(B)
    seq = torch.arange(B, device=dev).repeat_interleave(rows)
    slots = bt[seq, (pos // PAGE).long()] * PAGE + pos % PAGE
    qs = torch.arange(B + 1, **i32) * rows
    return BatchMeta(torch.randint(0, VOCAB, (B * rows,), **i32), pos, slots.int(), qs, torch.full((B,), ctx, **i32), bt, qs[1:] - 1,
                     rows, ctx, B, logits_all=rows == 1, host_lens=[(rows, ctx)] * B)


def model_numbers(cfg, dev, window: int, steps: int, warmup: int) -> dict:
    from oxidize_b200.models.transformer import Transformer

    model = Transformer(weights(cfg, dev), max_context=1 << 15)
    out = {"params_per_layer_m": round((cfg.param_count() - 2 * VOCAB * cfg.hidden_size) / LAYERS / 1e6, 1) if not cfg.is_mla else None}
    for B in (1, 64):
        meta = batch(B, 1, window + 1000, dev)
        kv = model.new_cache(meta.block_tables.numel(), PAGE, "bf16")
        for d in kv.data:
            d.normal_()
        step = lambda: model.greedy_tokens(meta, kv)
        if not cfg.is_mla:
            step = captured(step).replay
        ms = timed(step, steps, warmup)
        out[f"decode_b{B}"] = {"ms_per_step": round(ms, 4), "tok_s": round(B / ms * 1e3, 1)}
        del kv
    past = 2048 if window <= 1024 else 4096
    meta = batch(1, 2048, past + 2048, dev)
    kv = model.new_cache(meta.block_tables.numel(), PAGE, "bf16")
    for d in kv.data:
        d.normal_()
    ms = timed(lambda: model.greedy_tokens(meta, kv), max(4, steps // 4), warmup)
    out["prefill_2048"] = {"ms": round(ms, 3), "tok_s": round(2048 / ms * 1e3, 0)}
    return out


def kernel_numbers(width: int, heads: int, window: int, dev, steps: int) -> list:
    """The kernels of the layered model beside the like kernel of the grouped-query one: us, and the fraction of the slower
    of (bytes / copy bandwidth, products / bf16 peak).  Every case runs over several buffers in turn (larger than the L2)."""
    from oxidize_b200.engine.kv_pool import KVCache, KVCacheSpec
    from oxidize_b200.models.transformer import RopeState, Transformer
    from oxidize_b200.ops import cuda as C
    from oxidize_b200.ops import cuda_latent as CL
    from oxidize_b200.ops import ref

    gbs, tf = _peaks()
    rows = []
    cfg = layered(width, heads, window)
    spec, op_w = cfg.layer_specs[0].mixer, None
    model = Transformer(weights(cfg, dev), max_context=1 << 15)
    m = model.w.layers[0].mla
    op = CL.operands(m, spec, torch.bfloat16)
    rope = model.layer_ropes[0][0]
    nkv = max(1, heads // 4)
    grope = RopeState(ref.rope_inv_freq(128, 1e6, None, device=dev), "split_half", 1.0, heads, nkv, 128)

    def case(name, fns, nbytes, flops):
        g = captured(lambda: [f() for f in fns])
        us = timed(g.replay, max(8, steps), 3) / len(fns) * 1e3
        rows.append({"kernel": name, "us": round(us, 2), "of_roofline": round(max(nbytes / gbs / 1e3, flops / tf / 1e6) / us, 3),
                     "gb_s": round(nbytes / us / 1e3, 0), "tflop_s": round(flops / us / 1e6, 1)})

    for B, n, ctx in ((64, 1, window + 1000), (1, 1, window + 1000), (1, 2048, 2048 + (2048 if window <= 1024 else 4096))):
        T, L = B * n, 4 if B * n > 1 else 8
        meta = batch(B, n, ctx, dev)
        what = f"decode B={B}" if n == 1 else f"prefill {n}"
        keys = min(window, ctx)
        lat = KVCache(KVCacheSpec(L, 1, spec.row_dim, PAGE, "bf16", planes=1), meta.block_tables.numel(), dev)
        gqa = KVCache(KVCacheSpec(L, nkv, 128, PAGE, "bf16"), meta.block_tables.numel(), dev)
        for d in lat.data + gqa.data:
            d.normal_()
        span = B * min(ctx, keys + n - 1)
        # the attention step from rotated queries to per-head outputs: absorbed (the latent rows serve every head) or, for
        # long portions, over keys and values expanded per head
        xs = [torch.randn(T, heads * spec.qk_dim + RANK + ROT, device=dev).bfloat16() for _ in range(L)]
        qs = [torch.randn(T, heads, 128, device=dev).bfloat16() for _ in range(L)]
        pairs = T * heads * keys
        case(f"latent mixer without its projections, {what}",
             [lambda l=l: CL.latent_core(xs[l], m, spec, rope, meta, lat, l, 1e-5, op) for l in range(L)],
             span * spec.row_dim * 2 + (op.k.numel() + op.v.numel()) * 2 + T * (heads * (spec.qk_dim + VDIM)) * 2,
             2 * pairs * (DIM + ROT + VDIM) if n > 1 else 2 * pairs * (2 * RANK + ROT))
        case(f"grouped-query attention, {what}", [lambda l=l: C.paged_attention(qs[l], gqa, l, meta, 0.09, window) for l in range(L)],
             span * nkv * 512 + T * heads * 512, 4 * pairs * 128)
        if n == 1:
            q = torch.randn(T, heads, spec.row_dim, device=dev).bfloat16()
            o = torch.empty(heads, T, spec.latent_pad, dtype=torch.bfloat16, device=dev)
            case(f"latent attention kernel, {what}", [lambda l=l: CL.attention_mma(q, lat, l, meta, spec, m.sink, o) for l in range(L)],
                 span * spec.row_dim * 2 + T * heads * (spec.row_dim + RANK) * 2, 2 * pairs * (2 * RANK + ROT))
        R = max(1, min(64, (1 << 28) // (T * width * 12)))
        st = [torch.randn(T, width, device=dev) for _ in range(R)]
        ys = [torch.randn(T, width, device=dev).bfloat16() for _ in range(R)]
        rs = [torch.randn(T, width, device=dev).bfloat16() for _ in range(R)]
        w, b = torch.ones(width, device=dev), torch.zeros(width, device=dev)
        case(f"norm after the sum, {what}", [lambda i=i: CL.residual_norm(st[i], ys[i], 2.0, w, b, 1e-5, "layer", torch.bfloat16)
                                             for i in range(R)], T * width * 12, 0)
        case(f"add + RMS norm, {what}", [lambda i=i: C.add_rmsnorm(ys[i], rs[i], w, 1e-5) for i in range(R)], T * width * 8, 0)
        qn = torch.empty(heads, T, op.nope_ld, dtype=torch.bfloat16, device=dev)
        qa = torch.empty(T, heads, spec.row_dim, dtype=torch.bfloat16, device=dev)
        case(f"rotation + cache row (latent), {what}",
             [lambda l=l: CL.latent_prep(xs[l], m, spec, rope, meta, lat, l, 1e-5, op, q_nope=qn, q_rows=qa) for l in range(L)],
             T * (heads * spec.qk_dim + RANK + ROT) * 4, 0)
        qkv = [torch.randn(T, (heads + 2 * nkv) * 128, device=dev).bfloat16() for _ in range(L)]
        case(f"rotation + cache rows (grouped-query), {what}",
             [lambda l=l: C.qk_rope_kv_write(qkv[l], meta.positions, meta.slot_mapping, gqa, l, grope) for l in range(L)],
             T * (heads + 2 * nkv) * 128 * 4, 0)
        h = [torch.randn(T, width, device=dev).bfloat16() for _ in range(2)]
        up = model.w.layers
        case(f"up projection + squared relu, {what}", [lambda i=i: CL.linear_act(h[0], up[i].w_up, "relu2") for i in range(LAYERS)],
             4 * width * width * 2 + T * 5 * width * 2, 8 * T * width * width)
        case(f"up projection alone, {what}", [lambda i=i: C.linear(h[0], up[i].w_up.parts) for i in range(LAYERS)],
             4 * width * width * 2 + T * 5 * width * 2, 8 * T * width * width)
        del lat, gqa, xs, qs, st, ys, rs, qkv
    return rows


def main(args) -> int:
    if args.gpus != 1:
        raise SystemExit("--layered runs on one GPU")
    if args.design == "netovik":
        import netovik_bench

        return netovik_bench.main(args)
    if args.design == "pavatar":
        import pavatar_bench

        return pavatar_bench.main(args)
    if args.design == "sokirax":
        import sokirax_bench

        return sokirax_bench.main(args)
    from oxidize_b200.ops import cuda as C

    dev = torch.device("cuda", 0)
    torch.cuda.set_device(0)
    width, heads = (int(v) for v in args.layered.split("x"))
    gbs, tf = _peaks()
    for window in (1024, 4096):
        out = {"bench": "layered", "width": width, "heads": heads, "layers": LAYERS, "window": window, "dtype": "bf16",
               "data": "random weights and tokens", "peaks": {"gb_s": gbs, "bf16_tflop_s": tf}}
        for name, cfg in (("vefilix", layered(width, heads, window)), ("llama", uniform("llama", width, heads, window)),
                          ("deepseek2", uniform("deepseek2", width, heads, window))):
            out[name] = model_numbers(cfg, dev, window, args.steps, args.warmup)
            torch.cuda.empty_cache()
        out["kernels"] = kernel_numbers(width, heads, window, dev, args.steps)
        out["device_status"] = C.status()[0]
        print(json.dumps(out))
    return 0
