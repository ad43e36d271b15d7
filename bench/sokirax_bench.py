"""Throughput of Sokirax (attention and retention side by side, norms on both sides of every branch, dense and routed
feed-forward blocks) beside the closest uniform models at equal size, one GPU, random weights:

    python bench.py --layered 4096x32 --design sokirax --steps 32 --warmup 4

Three models of the same width, depth and window are timed: Sokirax, a grouped-query dense one (``llama``) whose feed-forward
blocks hold as many parameters as a Sokirax token passes through, and a routed one (``qwen3moe``, per-head q / k norm) with the
same experts in every layer.  Decode: captured steps replayed, every sequence past its window.  Prefill: portions of 2048 tokens
behind as many as the window and more.  Then the kernels that differ, each over buffers larger than the L2 in turn, against the
measured peaks."""
from __future__ import annotations

import json

import torch

from layered_bench import LAYERS, PAGE, VOCAB, _peaks, batch, captured, timed

DIM = 128
EXPERTS, TOP = 32, 4


def sizes(width: int):
    up = lambda n: (n + 127) // 128 * 128
    return up(8 * width // 3), up(width // 2), up(width)  # dense, expert, shared


def sokirax(width: int, heads: int, window: int):
    from oxidize_b200.models.config import (AttentionSpec, FeedForwardSpec, LayerSpec, MoESpec, ParallelSpec, RetentionSpec, RopeScaling,
                                            RotarySpec)
    from oxidize_b200.models.layered import layered_config

    ff, fe, fs = sizes(width)
    gated = lambda n: FeedForwardSpec(n, "silu", True)
    yarn = RotarySpec(64, 250000.0, RopeScaling("yarn", 4.0, 8192, 32.0, 1.0, ramp_limit=63, magnitude=1.1386))
    full = RotarySpec(DIM, 1e6)
    half = heads // 2
    att = AttentionSpec(heads, max(1, heads // 4), DIM, DIM, DIM ** -0.5, yarn, window, False, "head")
    par = ParallelSpec(AttentionSpec(half, max(1, half // 4), DIM, DIM, DIM ** -0.5, full, window, True, "full"),
                       RetentionSpec(half, DIM, DIM, [1 - 2.0 ** (-5 - 6 * i / half) for i in range(half)], full), 0.8, 0.5)
    moe = MoESpec(EXPERTS, TOP, gated(fe), gated(fs))
    kinds = [(att, gated(ff)), (att, moe), (par, gated(ff)), (par, moe)]
    return layered_config("sokirax", VOCAB, width, [LayerSpec(*kinds[i % 4]) for i in range(LAYERS)], 1e-5, "rms", norm_placement="sandwich")


def uniform(kind: str, width: int, heads: int, window: int):
    from oxidize_b200.models.config import ModelConfig

    ff, fe, fs = sizes(width)
    base = dict(vocab_size=VOCAB, hidden_size=width, n_layers=LAYERS, n_heads=heads, n_kv_heads=max(1, heads // 4), head_dim=DIM,
                context_length=1 << 16, sliding_window=window)
    if kind == "llama":
        return ModelConfig(arch="llama", ffn_size=(ff + TOP * fe + fs) // 2, **base)
    return ModelConfig(arch="qwen3moe", ffn_size=ff, qk_norm=True, n_experts=EXPERTS, n_experts_used=TOP, expert_ffn_size=fe,
                       n_shared_experts=1, shared_expert_ffn_size=fs, **base)


def with_slots(meta, first: int = 0):
    meta.state_slots = torch.arange(first, first + meta.num_seqs, dtype=torch.int32, device=meta.seq_lens.device)
    return meta


def model_numbers(cfg, dev, window: int, steps: int, warmup: int) -> dict:
    from oxidize_b200.models.transformer import Transformer
    from oxidize_b200.utils.synth import synth_weights

    model = Transformer(synth_weights(cfg, dev, "BF16", seed=0), max_context=1 << 15)
    out = {"params_m": round(cfg.param_count() / 1e6)}
    for B in (1, 64):
        meta = with_slots(batch(B, 1, window + 1000, dev))
        kv = model.new_cache(meta.block_tables.numel(), PAGE, "bf16", B)
        for d in kv.data:
            d.normal_()
        ms = timed(captured(lambda: model.greedy_tokens(meta, kv)).replay, steps, warmup)
        out[f"decode_b{B}"] = {"ms_per_step": round(ms, 4), "tok_s": round(B / ms * 1e3, 1)}
        del kv
    past = 2048 if window <= 1024 else 4096
    meta = with_slots(batch(1, 2048, past + 2048, dev))
    kv = model.new_cache(meta.block_tables.numel(), PAGE, "bf16", 1)
    for d in kv.data:
        d.normal_()
    ms = timed(lambda: model.greedy_tokens(meta, kv), max(4, steps // 4), warmup)
    out["prefill_2048"] = {"ms": round(ms, 3), "tok_s": round(2048 / ms * 1e3, 0)}
    return out


def kernel_numbers(width: int, heads: int, window: int, dev, steps: int) -> list:
    """us, and the fraction of the slower of (bytes / copy bandwidth, products / bf16 peak)."""
    from oxidize_b200.engine.kv_pool import KVCache, KVCacheSpec
    from oxidize_b200.models.transformer import RopeState
    from oxidize_b200.ops import cuda as C
    from oxidize_b200.ops import cuda_listed as CL
    from oxidize_b200.ops import ref

    gbs, tf = _peaks()
    rows = []
    specs = sokirax(width, heads, window).layer_specs
    att, par = specs[0].mixer, specs[2].mixer

    def case(name, fns, nbytes, flops):
        g = captured(lambda: [f() for f in fns])
        us = timed(g.replay, max(8, steps), 3) / len(fns) * 1e3
        rows.append({"kernel": name, "us": round(us, 2), "of_roofline": round(max(nbytes / gbs / 1e3, flops / tf / 1e6) / us, 3),
                     "gb_s": round(nbytes / us / 1e3, 0), "tflop_s": round(flops / us / 1e6, 1)})

    rope_of = lambda r: RopeState(ref.rope_inv_freq(r.dims, r.base, r.scaling, device=dev, dtype=torch.float64), "split_half",
                                  ref.rope_mscale(r.scaling), 0, 1, r.dims, 1 << 15)
    grope = RopeState(ref.rope_inv_freq(DIM, 1e6, None, device=dev), "split_half", 1.0, heads, max(1, heads // 4), DIM)
    one = lambda n: torch.ones(n, device=dev)
    for B, n, ctx in ((64, 1, window + 1000), (1, 1, window + 1000), (1, 2048, 2048 + (2048 if window <= 1024 else 4096))):
        T, L = B * n, 4 if B * n > 1 else 8
        what = f"decode B={B}" if n == 1 else f"prefill {n}"
        meta = with_slots(batch(B, n, ctx, dev))
        keys = min(window, ctx)
        span = B * min(ctx, keys + n - 1)
        G = att.kv_heads
        kv = KVCache(KVCacheSpec(L, G, DIM, PAGE, "bf16"), meta.block_tables.numel(), dev)
        for d in kv.data:
            d.normal_()
        qs = [torch.randn(T, heads, DIM, device=dev).bfloat16() for _ in range(L)]
        out = torch.empty(T, att.out_dim, dtype=torch.bfloat16, device=dev)
        nb, fl = span * G * 2 * DIM * 2 + T * heads * DIM * 4, 4 * T * heads * keys * DIM
        sink = torch.randn(heads, device=dev)
        case(f"attention (sokirax, with sinks), {what}", [lambda l=l: CL.attention(qs[l], kv, l, meta, att, sink, out, 0.8) for l in range(L)],
             nb, fl)
        case(f"attention (llama), {what}", [lambda l=l: C.paged_attention(qs[l], kv, l, meta, att.scale, window) for l in range(L)], nb, fl)
        zs = [torch.randn(T, att.proj_dim, device=dev).bfloat16() for _ in range(L)]
        rope = rope_of(att.rotary)
        qn, kn = one(DIM), one(DIM)
        nb = T * (heads + 2 * G) * DIM * 4
        case(f"head norm + rotation + cache rows (sokirax), {what}",
             [lambda l=l: CL.head_prep(zs[l], qn, kn, att, rope, meta, kv, l, 1e-5) for l in range(L)], nb, 0)
        import dataclasses

        fulls, fq, fk = dataclasses.replace(att, qk_norm="full"), one(heads * DIM), one(G * DIM)
        case(f"full norm + rotation + cache rows (sokirax), {what}",
             [lambda l=l: CL.head_prep(zs[l], fq, fk, fulls, rope, meta, kv, l, 1e-5) for l in range(L)], nb, 0)
        case(f"head norm + rotation + cache rows (qwen3moe), {what}",
             [lambda l=l: C.qk_rope_kv_write(zs[l], meta.positions, meta.slot_mapping, kv, l, grope, qn, kn, 1e-5) for l in range(L)], nb, 0)
        del kv, qs, zs
        r = par.right
        H, K, V = r.state_shape
        zr = [torch.randn(T, r.proj_dim, device=dev).bfloat16() for _ in range(L)]
        st = [torch.zeros(B, H, K, V, device=dev) for _ in range(max(L, 1 + (1 << 28) // (B * H * K * V * 4)))][:16]
        dec = torch.tensor(r.decay, device=dev)
        ro = torch.empty(T, r.out_dim, dtype=torch.bfloat16, device=dev)
        nb = B * H * K * V * 8 + T * H * (2 * K + 3 * V) * 2
        # products of a chunk of 64: scores and their values (half of the square), state to outputs, values to state
        fl = 2 * T * H * ((64 // 2) * (K + V) + 2 * K * V) if n > 1 else 4 * T * H * K * V
        rr = rope_of(r.rotary)
        case(f"retention (rotation to gated output), {what}",
             [lambda l=l: CL.retention(zr[l % L], r, rr, meta, st[l], dec, 1e-5, ro, 0.5) for l in range(len(st))], nb, fl)
        del zr, st
        R = max(1, min(64, (1 << 28) // (T * width * 14)))
        xs = [torch.randn(T, width, device=dev) for _ in range(R)]
        ys = [torch.randn(T, width, device=dev).bfloat16() for _ in range(R)]
        rs = [torch.randn(T, width, device=dev).bfloat16() for _ in range(R)]
        w = one(width)
        case(f"norms on both sides of a branch (sokirax), {what}",
             [lambda i=i: CL.branch_norm(xs[i], ys[i], w, w, 1e-5, torch.bfloat16) for i in range(R)], T * width * 12, 0)
        case(f"add + RMS norm (llama), {what}", [lambda i=i: C.add_rmsnorm(ys[i], rs[i], w, 1e-5) for i in range(R)], T * width * 8, 0)
        from oxidize_b200.models.weights import QTensor

        rw = [QTensor("BF16", torch.randn(EXPERTS, width, device=dev).bfloat16(), (EXPERTS, width)) for _ in range(R)]
        nb = T * width * 2 + EXPERTS * width * 2 + T * EXPERTS * 4
        case(f"router logits, float32 (sokirax), {what}", [lambda i=i: CL.router_logits(ys[i], rw[i]) for i in range(R)], nb,
             2 * T * width * EXPERTS)
        case(f"router logits, bf16 (qwen3moe), {what}", [lambda i=i: C.linear(ys[i], [rw[i]]).float() for i in range(R)], nb,
             2 * T * width * EXPERTS)
        del xs, ys, rs, rw
        torch.cuda.empty_cache()
    return rows


def main(args) -> int:
    from oxidize_b200.ops import cuda as C

    dev = torch.device("cuda", 0)
    torch.cuda.set_device(0)
    width, heads = (int(v) for v in args.layered.split("x"))
    gbs, tf = _peaks()
    for window in (1024, 4096):
        out = {"bench": "layered", "design": "sokirax", "width": width, "heads": heads, "layers": LAYERS, "window": window,
               "dtype": "bf16", "data": "random weights and tokens", "peaks": {"gb_s": gbs, "bf16_tflop_s": tf}}
        for name, cfg in (("sokirax", sokirax(width, heads, window)), ("llama", uniform("llama", width, heads, window)),
                          ("qwen3moe", uniform("qwen3moe", width, heads, window))):
            out[name] = model_numbers(cfg, dev, window, args.steps, args.warmup)
            torch.cuda.empty_cache()
        out["kernels"] = kernel_numbers(width, heads, window, dev, args.steps)
        out["device_status"] = C.status()[0]
        print(json.dumps(out))
    return 0
