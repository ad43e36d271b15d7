"""Throughput of Netovik (RWKV time mixing, attention on mixed head scores, norms in groups on the branches' outputs, a weighted
sum of all earlier results after every layer, dense and routed gated feed-forward blocks) beside the closest models at equal size,
one GPU, random weights:

    python bench.py --layered 4096x32 --design netovik --steps 32 --warmup 4

Three models of the same width, depth, window and feed-forward blocks are timed: Netovik, Sokirax (retention layers and
grouped-query attention with a norm per head) and a grouped-query one (``qwen3moe``).  Decode: captured steps replayed, every
sequence past its window.  Prefill: portions of 2048 tokens behind as many as the window and more.  Then the kernels that differ,
each over buffers larger than the L2 in turn, against the measured peaks."""
from __future__ import annotations

import dataclasses
import json

import torch

from layered_bench import LAYERS, PAGE, VOCAB, _peaks, batch, captured, timed
from sokirax_bench import DIM, EXPERTS, TOP, model_numbers, sizes, with_slots

KEEP, RANK, BUCKETS, FAR = 4, 64, 32, 128


def blocks(width: int):
    """Feed-forward blocks of the layers: dense, then routed experts, and so on."""
    from oxidize_b200.models.config import FeedForwardSpec, MoESpec

    ff, fe, _ = sizes(width)
    moe = MoESpec(EXPERTS, TOP, FeedForwardSpec(fe, "silu", True))
    return [FeedForwardSpec(ff, "silu", True), moe], dataclasses.replace(moe, expert_weights_norm=False)


def attention_spec(heads: int, window: int):
    from oxidize_b200.models.config import AttentionSpec

    return AttentionSpec(heads, max(1, heads // 4), DIM, DIM, DIM ** -0.5, None, window, qk_norm="unit", bias=True, keep_first=KEEP,
                         softcap=50.0, bias_rows=BUCKETS, bias_max=FAR, talk=True, unit_sink=True, shared_kv=True)


def netovik(width: int, heads: int, window: int):
    from oxidize_b200.models.config import LayerSpec, WkvSpec
    from oxidize_b200.models.layered import layered_config

    (dense, _), moe = blocks(width)
    kinds = [(WkvSpec(heads, DIM, RANK, width), dense), (attention_spec(heads, window), moe), (WkvSpec(heads, DIM, RANK, width), moe),
             (attention_spec(heads, window), dense)]
    cfg = layered_config("netovik", VOCAB, width, [LayerSpec(*kinds[i % 4]) for i in range(LAYERS)], 1e-5, "rms", norm_placement="output")
    cfg.norm_groups, cfg.depth_average, cfg.embedding_scale, cfg.tie_embeddings = 2, True, 8.0, True
    return cfg


def sokirax(width: int, heads: int, window: int):
    from oxidize_b200.models.config import AttentionSpec, LayerSpec, RetentionSpec, RotarySpec
    from oxidize_b200.models.layered import layered_config

    (dense, moe), _ = blocks(width)
    full = RotarySpec(DIM, 1e6)
    ret = RetentionSpec(heads, DIM, DIM, [1 - 2.0 ** (-5 - 6 * i / heads) for i in range(heads)], full)
    att = AttentionSpec(heads, max(1, heads // 4), DIM, DIM, DIM ** -0.5, full, window, False, "head")
    kinds = [(ret, dense), (att, moe), (ret, moe), (att, dense)]
    return layered_config("sokirax", VOCAB, width, [LayerSpec(*kinds[i % 4]) for i in range(LAYERS)], 1e-5, "rms", norm_placement="sandwich")


def qwen3moe(width: int, heads: int, window: int):
    from oxidize_b200.models.config import ModelConfig

    return ModelConfig(arch="qwen3moe", vocab_size=VOCAB, hidden_size=width, n_layers=LAYERS, n_heads=heads, n_kv_heads=max(1, heads // 4),
                       head_dim=DIM, context_length=1 << 16, ffn_size=sizes(width)[0], qk_norm=True, n_experts=EXPERTS,
                       n_experts_used=TOP, expert_ffn_size=sizes(width)[1], sliding_window=window)


def kernel_numbers(width: int, heads: int, window: int, dev, steps: int) -> list:
    """us, and the fraction of the slower of (bytes / copy bandwidth, products / bf16 peak)."""
    from oxidize_b200 import ops
    from oxidize_b200.engine.kv_pool import KVCache, KVCacheSpec
    from oxidize_b200.models.transformer import RopeState
    from oxidize_b200.ops import cuda as C
    from oxidize_b200.ops import cuda_joint as CJ
    from oxidize_b200.ops import cuda_latent as CLat
    from oxidize_b200.ops import cuda_listed as CL
    from oxidize_b200.ops import cuda_wkv as CW
    from oxidize_b200.ops import ref
    from oxidize_b200.utils.synth import synth_weights

    gbs, tf = _peaks()
    rows = []

    def case(name, fns, nbytes, flops):
        g = captured(lambda: [f() for f in fns])
        us = timed(g.replay, max(8, steps), 3) / len(fns) * 1e3
        rows.append({"kernel": name, "us": round(us, 2), "of_roofline": round(max(nbytes / gbs / 1e3, flops / tf / 1e6) / us, 3),
                     "gb_s": round(nbytes / us / 1e3, 0), "tflop_s": round(flops / us / 1e6, 1)})

    cfg, like = netovik(width, heads, window), sokirax(width, heads, window)
    w = synth_weights(dataclasses.replace(cfg, layer_specs=cfg.layer_specs[:2], n_layers=2), dev, "BF16", seed=0).layers
    wkv, att = cfg.layer_specs[0].mixer, cfg.layer_specs[1].mixer
    ret, latt = like.layer_specs[0].mixer, like.layer_specs[1].mixer
    full = RopeState(ref.rope_inv_freq(DIM, 1e6, None, device=dev, dtype=torch.float64), "split_half", 1.0, 0, 1, DIM, 1 << 15)
    one = lambda n: torch.ones(n, device=dev)
    for B, n, ctx in ((64, 1, window + 1000), (1, 1, window + 1000), (1, 2048, 2048 + (2048 if window <= 1024 else 4096))):
        T, L = B * n, 4 if B * n > 1 else 8
        what = f"decode B={B}" if n == 1 else f"prefill {n}"
        meta = with_slots(batch(B, n, ctx, dev))
        rnd = lambda *s: torch.randn(*s, device=dev).bfloat16()
        # ---- recurrences
        H, K, V = wkv.state_shape
        N = max(1, min(16, (1 << 28) // (B * H * K * V * 4) + 1))
        st = [torch.zeros(B, H, K, V, device=dev) for _ in range(N)]
        zs, dec = [rnd(T, 4 * H * K) for _ in range(L)], [-0.1 * torch.rand(T, H * K, device=dev) for _ in range(L)]
        out = torch.empty(T, H * V, dtype=torch.bfloat16, device=dev)
        lw = w[0].wkv
        nb = B * H * K * V * 8 + T * H * K * (8 + 4 + 2)
        case(f"RWKV recurrence ({H} heads), {what}", [lambda l=l: CW.wkv(zs[l % L], dec[l % L], lw, wkv, meta, st[l], 1e-5, out) for l in range(N)], nb,
             4 * T * H * K * V)
        decay = torch.tensor(ret.decay, device=dev)
        nb = B * H * K * V * 8 + T * H * K * 10
        case(f"retention ({H} heads), {what}", [lambda l=l: CL.retention(zs[l % L], ret, full, meta, st[l], decay, 1e-5, out, 1.0) for l in range(N)],
             nb, 4 * T * H * K * V)
        del st, zs, dec
        R = max(1, min(32, (1 << 28) // (T * width * 14)))
        xs = [torch.randn(T, width, device=dev) for _ in range(R)]
        win = torch.zeros(B, 1, width, device=dev)
        case(f"token shift, {what}", [lambda i=i: CW.token_shift(xs[i], lw.mu, meta, win, torch.bfloat16) for i in range(R)], T * width * 14, 0)
        low = [rnd(T, RANK) for _ in range(4)]
        case(f"decays, {what}", [lambda i=i: CW.log_decay(low[i], lw) for i in range(4)], T * (H * K * 4 + RANK * 2) + H * K * RANK * 2, 2 * T * H * K * RANK)
        mixes, z = [rnd(5, T, width) for _ in range(2)], torch.empty(T, 4 * H * K, dtype=torch.bfloat16, device=dev)
        nb, fl = 4 * H * K * width * 2 + T * (4 * width + 4 * H * K) * 2, 8 * T * H * K * width
        case(f"r, k, v, gate projections of four inputs, {what}",
             [lambda i=i: CLat.batched(mixes[i][:4], lw.proj, z, H * K, 4 * H * K) for i in range(2)], nb, fl)
        from oxidize_b200.models.layered import dense_qtensor

        four = dense_qtensor(lw.proj.reshape(4 * H * K, -1))
        case(f"the same four of one input, {what}", [lambda i=i: C.linear(mixes[i][0], [four]) for i in range(2)], nb - 3 * T * width * 2, fl)
        del mixes, z
        # ---- attention and what surrounds it
        G = att.kv_heads
        kv = KVCache(KVCacheSpec(L, *[att.cache_shape[i] for i in (0, 2)], PAGE, "bf16", planes=1), meta.block_tables.numel(), dev)
        lkv = KVCache(KVCacheSpec(L, G, DIM, PAGE, "bf16"), meta.block_tables.numel(), dev)
        for d in kv.data + lkv.data:
            d.normal_()
        qs, zs = [rnd(T, heads, DIM) for _ in range(L)], [rnd(T, latt.qkv_dim) for _ in range(L)]
        out = torch.empty(T, heads * DIM, dtype=torch.bfloat16, device=dev)
        seen = min(ctx, window + n - 1)
        pairs = T * heads * min(window, ctx)
        a1 = w[1]
        case(f"attention on mixed scores (one row per key), {what}",
             [lambda l=l: CJ.attention(qs[l], kv, l, meta, att, a1.score_bias, a1.score_mix, a1.sink, out, 1.0) for l in range(L)],
             B * seen * G * (DIM + 8) * 2 + T * heads * DIM * 4, 4 * pairs * DIM)
        case(f"attention (sokirax), {what}", [lambda l=l: CL.attention(qs[l], lkv, l, meta, latt, None, out, 1.0) for l in range(L)],
             B * seen * G * 2 * DIM * 2 + T * heads * DIM * 4, 4 * pairs * DIM)
        qn, kn = one(DIM), one(DIM)
        case(f"unit norms + cache rows, {what}", [lambda l=l: CL.head_prep(zs[l], None, None, att, None, meta, kv, l, 1e-5) for l in range(L)],
             T * (heads + G) * DIM * 4, 0)
        case(f"head norm + rotation + cache rows (sokirax), {what}",
             [lambda l=l: CL.head_prep(zs[l], qn, kn, latt, full, meta, lkv, l, 1e-5) for l in range(L)], T * (heads + 2 * G) * DIM * 4, 0)
        del kv, lkv, qs, zs
        # ---- norms
        ys, g = [rnd(T, width) for _ in range(R)], one(width)
        er, idx = rnd(T * TOP, width), torch.randperm(T * TOP, device=dev).reshape(T, TOP).int()
        routed = ops.RoutedRows(er, idx, torch.rand(T, TOP, device=dev))
        case(f"grouped norm + sum, {what}", [lambda i=i: CL.add_normed(xs[i], ys[i], g, 2, 1e-5, torch.bfloat16) for i in range(R)], T * width * 12, 0)
        for layer in (0, LAYERS - 1):
            streams, depth = ops.DepthStreams(xs[0], LAYERS), one(layer + 2) / (layer + 2)

            def run(i):
                streams.n = layer
                return CL.add_normed(xs[i], routed, g, 2, 1e-5, torch.bfloat16, streams, depth)

            case(f"grouped norm + experts' sum + depth average, layer {layer}, {what}", [lambda i=i: run(i) for i in range(R)],
                 T * width * (4 + 2 * TOP + 4 + 4 + 2 + 4 + 4 * layer), 0)
        case(f"norms on both sides of a branch (sokirax), {what}",
             [lambda i=i: CL.branch_norm(xs[i], ys[i], g, g, 1e-5, torch.bfloat16) for i in range(R)], T * width * 12, 0)
        del xs, ys, er
        torch.cuda.empty_cache()
    return rows


def main(args) -> int:
    from oxidize_b200.ops import cuda as C

    dev = torch.device("cuda", 0)
    torch.cuda.set_device(0)
    width, heads = (int(v) for v in args.layered.split("x"))
    gbs, tf = _peaks()
    for window in (1024, 4096):
        out = {"bench": "layered", "design": "netovik", "width": width, "heads": heads, "layers": LAYERS, "window": window, "dtype": "bf16",
               "data": "random weights and tokens", "peaks": {"gb_s": gbs, "bf16_tflop_s": tf}}
        for name, make in (("netovik", netovik), ("sokirax", sokirax), ("qwen3moe", qwen3moe)):
            out[name] = model_numbers(make(width, heads, window), dev, window, args.steps, args.warmup)
            torch.cuda.empty_cache()
        out["kernels"] = kernel_numbers(width, heads, window, dev, args.steps)
        out["device_status"] = C.status()[0]
        print(json.dumps(out))
    return 0
