"""Throughput of Pavatar (gated delta rule, unrotated attention with mixed values, both kinds side by side, routed squared-relu
experts, one norm for mixer and experts) beside the closest models at equal size, one GPU, random weights:

    python bench.py --layered 4096x32 --design pavatar --steps 32 --warmup 4

Three models of the same width, depth and routed experts are timed: Pavatar, Sokirax without windows (attention, and retention
beside attention) and a grouped-query one (``qwen3moe``).  Decode: captured steps replayed.  Prefill: portions of 2048 tokens
behind as many and more.  Then the kernels that differ, each over buffers larger than the L2 in turn, against the measured
peaks."""
from __future__ import annotations

import json

import torch

from layered_bench import LAYERS, PAGE, VOCAB, _peaks, batch, captured, timed
from sokirax_bench import DIM, EXPERTS, TOP, sizes, with_slots

RANK = 128


def expert_size(width: int) -> int:
    """Two matrices per expert instead of a gated one's three."""
    return sizes(width)[1] * 3 // 2


def pavatar(width: int, heads: int):
    from oxidize_b200.models.config import AttentionSpec, DeltaSpec, FeedForwardSpec, LayerSpec, MoESpec, ParallelSpec, RotarySpec
    from oxidize_b200.models.layered import layered_config

    half = heads // 2
    moe = MoESpec(EXPERTS, TOP, FeedForwardSpec(expert_size(width), "relu2"), expert_weights_scale=2.0, correction=True)
    att = AttentionSpec(heads, max(1, heads // 4), DIM, DIM, DIM ** -0.5, None, bias=True, temp_coef=0.1, temp_every=8192.0, v_mix=True,
                        gate="head")
    par = ParallelSpec(AttentionSpec(half, max(1, half // 4), DIM, DIM, DIM ** -0.5, RotarySpec(DIM, 1e6), qk_norm="head", gate="value"),
                       DeltaSpec(half, half, DIM, DIM, 4, RANK, RANK), 0.5, 0.5, norms=True)
    kinds = [DeltaSpec(heads, half, DIM, DIM, 4), att, par, att]
    cfg = layered_config("pavatar", VOCAB, width, [LayerSpec(kinds[i % 4], moe) for i in range(LAYERS)], 1e-5, "rms", norm_placement="parallel")
    cfg.embedding_scale, cfg.final_softcap, cfg.tie_embeddings = 8.0, 50.0, True
    return cfg


def sokirax(width: int, heads: int):
    from oxidize_b200.models.config import AttentionSpec, FeedForwardSpec, LayerSpec, MoESpec, ParallelSpec, RetentionSpec, RotarySpec
    from oxidize_b200.models.layered import layered_config

    half, full = heads // 2, RotarySpec(DIM, 1e6)
    moe = MoESpec(EXPERTS, TOP, FeedForwardSpec(sizes(width)[1], "silu", True))
    ret = lambda n: RetentionSpec(n, DIM, DIM, [1 - 2.0 ** (-5 - 6 * i / n) for i in range(n)], full)
    att = AttentionSpec(heads, max(1, heads // 4), DIM, DIM, DIM ** -0.5, full, 0, False, "head")
    par = ParallelSpec(AttentionSpec(half, max(1, half // 4), DIM, DIM, DIM ** -0.5, full, 0, True, "full"), ret(half), 0.8, 0.5)
    kinds = [ret(heads), att, par, att]
    return layered_config("sokirax", VOCAB, width, [LayerSpec(kinds[i % 4], moe) for i in range(LAYERS)], 1e-5, "rms", norm_placement="sandwich")


def qwen3moe(width: int, heads: int):
    from oxidize_b200.models.config import ModelConfig

    return ModelConfig(arch="qwen3moe", vocab_size=VOCAB, hidden_size=width, n_layers=LAYERS, n_heads=heads, n_kv_heads=max(1, heads // 4),
                       head_dim=DIM, context_length=1 << 16, ffn_size=sizes(width)[0], qk_norm=True, n_experts=EXPERTS,
                       n_experts_used=TOP, expert_ffn_size=sizes(width)[1])


def model_numbers(cfg, dev, ctx: int, past: int, steps: int, warmup: int) -> dict:
    from oxidize_b200.models.transformer import Transformer
    from oxidize_b200.utils.synth import synth_weights

    model = Transformer(synth_weights(cfg, dev, "BF16", seed=0), max_context=1 << 15)
    out = {"params_m": round(cfg.param_count() / 1e6)}
    for B in (1, 64):
        meta = with_slots(batch(B, 1, ctx, dev))
        kv = model.new_cache(meta.block_tables.numel(), PAGE, "bf16", B)
        for d in kv.data:
            d.normal_()
        ms = timed(captured(lambda: model.greedy_tokens(meta, kv)).replay, steps, warmup)
        out[f"decode_b{B}"] = {"ms_per_step": round(ms, 4), "tok_s": round(B / ms * 1e3, 1)}
        del kv
    meta = with_slots(batch(1, 2048, past + 2048, dev))
    kv = model.new_cache(meta.block_tables.numel(), PAGE, "bf16", 1)
    for d in kv.data:
        d.normal_()
    ms = timed(lambda: model.greedy_tokens(meta, kv), max(4, steps // 4), warmup)
    out["prefill_2048"] = {"ms": round(ms, 3), "tok_s": round(2048 / ms * 1e3, 0)}
    return out


def kernel_numbers(width: int, heads: int, ctx: int, past: int, dev, steps: int) -> list:
    """us, and the fraction of the slower of (bytes / copy bandwidth, products / bf16 peak)."""
    from oxidize_b200 import ops
    from oxidize_b200.engine.kv_pool import KVCache, KVCacheSpec
    from oxidize_b200.models.transformer import RopeState
    from oxidize_b200.ops import cuda as C
    from oxidize_b200.ops import cuda_delta as CD
    from oxidize_b200.ops import cuda_listed as CL
    from oxidize_b200.ops import ref
    from oxidize_b200.utils.synth import synth_weights

    gbs, tf = _peaks()
    rows = []

    def case(name, fns, nbytes, flops):
        g = captured(lambda: [f() for f in fns])
        us = timed(g.replay, max(8, steps), 3) / len(fns) * 1e3
        rows.append({"kernel": name, "us": round(us, 2), "of_roofline": round(max(nbytes / gbs / 1e3, flops / tf / 1e6) / us, 3),
                     "gb_s": round(nbytes / us / 1e3, 0), "tflop_s": round(flops / us / 1e6, 1)})

    import dataclasses

    cfg, like = pavatar(width, heads), sokirax(width, heads)
    w = synth_weights(dataclasses.replace(cfg, layer_specs=cfg.layer_specs[:4], n_layers=4), dev, "BF16", seed=0).layers
    wl = synth_weights(dataclasses.replace(like, layer_specs=like.layer_specs[1:2], n_layers=1), dev, "BF16", seed=0).layers[0]
    dlt, att, par = cfg.layer_specs[0].mixer, cfg.layer_specs[1].mixer, cfg.layer_specs[2].mixer
    ret, latt = like.layer_specs[0].mixer, like.layer_specs[1].mixer
    moe, lmoe = cfg.layer_specs[0].ffn, like.layer_specs[0].ffn
    full = RopeState(ref.rope_inv_freq(DIM, 1e6, None, device=dev, dtype=torch.float64), "split_half", 1.0, 0, 1, DIM, 1 << 15)
    one = lambda n: torch.ones(n, device=dev)
    for B, n, c in ((64, 1, ctx), (1, 1, ctx), (1, 2048, past + 2048)):
        T, L = B * n, 4 if B * n > 1 else 8
        what = f"decode B={B}" if n == 1 else f"prefill {n}"
        meta = with_slots(batch(B, n, c, dev))
        rnd = lambda *s: torch.randn(*s, device=dev).bfloat16()
        # ---- recurrences; products of a step: S^T k, k u^T and S^T q
        for name, spec, lw in (("delta rule, decay per head", dlt, w[0]), ("delta rule, decay per channel", par.right, w[2])):
            H, K, V = spec.state_shape
            zs = [rnd(T, spec.proj_dim) for _ in range(L)]
            N = max(1, min(16, (1 << 28) // (B * H * K * V * 4) + 1))
            st = [torch.zeros(B, H, K, V, device=dev) for _ in range(N)]
            win = [torch.zeros(B, *spec.window_shape, device=dev) for _ in range(N)]
            out = torch.empty(T, spec.out_dim, dtype=torch.bfloat16, device=dev)
            nb = B * H * K * V * 8 + T * (spec.proj_dim + spec.out_dim) * 2
            case(f"{name} ({H} heads), {what}",
                 [lambda l=l: CD.delta_rule(zs[l % L], lw.delta, spec, meta, st[l], win[l], 1e-5, out) for l in range(N)], nb, 6 * T * H * K * V)
            r = dataclasses.replace(ret, heads=H, decay=ret.decay[:H])
            zr, dec = [rnd(T, r.proj_dim) for _ in range(L)], torch.tensor(r.decay, device=dev)
            nb = B * H * K * V * 8 + T * (r.proj_dim + r.out_dim) * 2
            case(f"retention ({H} heads), {what}", [lambda l=l: CL.retention(zr[l % L], r, full, meta, st[l], dec, 1e-5, out, 1.0) for l in range(N)],
                 nb, 4 * T * H * K * V)
            del st, win, zs, zr
        # ---- attention and what surrounds it
        G = att.kv_heads
        kv = KVCache(KVCacheSpec(L, G, DIM, PAGE, "bf16"), meta.block_tables.numel(), dev)
        for d in kv.data:
            d.normal_()
        qs, zs = [rnd(T, heads, DIM) for _ in range(L)], [rnd(T, att.proj_dim) for _ in range(L)]
        out = torch.empty(T, att.out_dim, dtype=torch.bfloat16, device=dev)
        keys = c - (n - 1) / 2
        nb, fl = B * c * G * 2 * DIM * 2 + T * heads * DIM * 4, 4 * T * heads * keys * DIM
        gates = [z[:, att.qkv_dim :] for z in zs]
        vgate = [rnd(T, heads * DIM) for _ in range(L)]
        val = dataclasses.replace(att, gate="value")
        case(f"attention, gate per head (pavatar), {what}",
             [lambda l=l: CL.attention(qs[l], kv, l, meta, att, None, out, 1.0, gates[l]) for l in range(L)], nb, fl)
        case(f"attention, gate per value (pavatar), {what}",
             [lambda l=l: CL.attention(qs[l], kv, l, meta, val, None, out, 1.0, vgate[l]) for l in range(L)], nb + T * heads * DIM * 2, fl)
        case(f"attention (sokirax), {what}", [lambda l=l: CL.attention(qs[l], kv, l, meta, latt, None, out, 1.0) for l in range(L)], nb, fl)
        first, mix, qn, kn = rnd(T, G, DIM), 0.5 * one(1), one(DIM), one(DIM)
        nb = T * (heads + 2 * G) * DIM * 4
        case(f"temperature + mixed values + cache rows (pavatar), {what}",
             [lambda l=l: CL.head_prep(zs[l], None, None, att, None, meta, kv, l, 1e-5, first, mix) for l in range(L)], nb + T * G * DIM * 2, 0)
        case(f"head norm + rotation + cache rows (sokirax), {what}",
             [lambda l=l: CL.head_prep(zs[l], qn, kn, latt, full, meta, kv, l, 1e-5) for l in range(L)], nb, 0)
        del kv, qs, zs, vgate
        # ---- norms and experts
        R = max(1, min(32, (1 << 28) // (T * width * 14)))
        xs, ys, fs = ([f() for _ in range(R)] for f in (lambda: torch.randn(T, width, device=dev), lambda: rnd(T, width), lambda: rnd(T, width)))
        er = rnd(T * TOP, width)
        idx = torch.randperm(T * TOP, device=dev).reshape(T, TOP).int()
        routed, g = ops.RoutedRows(er, idx, torch.rand(T, TOP, device=dev)), one(width)
        case(f"both branches, experts' sum, next norm (pavatar), {what}",
             [lambda i=i: CL.joint_norm(xs[i], ys[i], routed, g, 1e-5, torch.bfloat16) for i in range(R)], T * width * (12 + 2 * TOP), 0)
        case(f"two normed outputs, experts' sum, next norm (pavatar), {what}",
             [lambda i=i: CL.joint_norm(xs[i], ops.NormedPair(ys[i], fs[i], g, g, 0.5, 0.5), routed, g, 1e-5, torch.bfloat16) for i in range(R)],
             T * width * (14 + 2 * TOP), 0)
        case(f"norms on both sides of a branch (sokirax), {what}",
             [lambda i=i: CL.branch_norm(xs[i], ys[i], g, g, 1e-5, torch.bfloat16) for i in range(R)], T * width * 12, 0)
        active = min(EXPERTS, T * TOP)
        fe, fl = expert_size(width), sizes(width)[1]
        case(f"experts, squared relu (pavatar), {what}", [lambda i=i: CL.moe_ffn(ys[i % R], w[0], moe, False) for i in range(2)],
             active * 2 * width * fe * 2 + T * width * (2 + 2 * TOP), 4 * T * TOP * width * fe)
        case(f"experts, gated (sokirax), {what}", [lambda i=i: CL.moe_ffn(ys[i % R], wl, lmoe) for i in range(2)],
             active * 3 * width * fl * 2 + T * width * (4 + 2 * TOP), 6 * T * TOP * width * fl)
        del xs, ys, fs, er
        torch.cuda.empty_cache()
    return rows


def main(args) -> int:
    from oxidize_b200.ops import cuda as C

    dev = torch.device("cuda", 0)
    torch.cuda.set_device(0)
    width, heads = (int(v) for v in args.layered.split("x"))
    gbs, tf = _peaks()
    for ctx, past in ((2048, 2048), (8192, 6144)):
        out = {"bench": "layered", "design": "pavatar", "width": width, "heads": heads, "layers": LAYERS, "context": ctx, "past": past,
               "dtype": "bf16", "data": "random weights and tokens", "peaks": {"gb_s": gbs, "bf16_tflop_s": tf}}
        for name, make in (("pavatar", pavatar), ("sokirax", sokirax), ("qwen3moe", qwen3moe)):
            out[name] = model_numbers(make(width, heads), dev, ctx, past, args.steps, args.warmup)
            torch.cuda.empty_cache()
        out["kernels"] = kernel_numbers(width, heads, ctx, past, dev, args.steps)
        out["device_status"] = C.status()[0]
        print(json.dumps(out))
    return 0
