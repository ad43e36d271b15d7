"""The mechanisms of listed layers with grouped-query attention and retention, one at a time: norms on both sides of a branch,
head norms and rotation, attention (window edges, page borders, sink, long portions), retention (steps, chunks, segments, state
slots), routed experts, configuration checks."""
import itertools
import json
import os

import numpy as np
import pytest
import torch

import sokirax_plain as plain
from oxidize_b200 import ops
from oxidize_b200.engine.kv_pool import KVCache, KVCacheSpec, OutOfBlocks, StateSlots
from oxidize_b200.engine.llm import LLM, EngineConfig
from oxidize_b200.models.config import (AttentionSpec, FeedForwardSpec, LayerSpec, MoESpec, ParallelSpec, RetentionSpec, RotarySpec,
                                        UnsupportedArchitecture)
from oxidize_b200.models.layered import gated_pair, listed_experts, pad_heads
from oxidize_b200.models.transformer import BatchMeta, RopeState
from oxidize_b200.models.weights import LayerWeights, LinearWeight, QTensor
from oxidize_b200.ops import ref as opref

gpu = pytest.mark.gpu
CPU = pytest.param("cpu", torch.float32, id="cpu")
F32 = pytest.param("cuda", torch.float32, id="gpu32", marks=gpu)
B16 = pytest.param("cuda", torch.bfloat16, id="gpu16", marks=gpu)


@pytest.fixture(autouse=True)
def _status():
    yield
    if torch.cuda.is_available():
        from oxidize_b200.ops import cuda as C

        assert C.status()[0] == 0


def rel(a, b):
    a, b = torch.as_tensor(a).double().cpu(), torch.as_tensor(b).double().cpu()
    return float((a - b).norm() / (b.norm() + 1e-30))


def worst_row(got, want):
    """Largest distance of a row from its like, in units of the rows' root mean square."""
    d = (torch.as_tensor(got).double().cpu() - torch.as_tensor(want).double()).pow(2).mean(-1).sqrt()
    return float(d.max() / torch.as_tensor(want).double().pow(2).mean().sqrt())


# --------------------------------------------------------------------------- norms
@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("T,H", [(1, 4), (5, 96), (3, 257), (7, 4096), (2, 6144), (600, 2048), (2, 10002)])
def test_norms_on_both_sides_of_a_branch(device, dtype, T, H):
    g = torch.Generator().manual_seed(H)
    res, y = torch.randn(T, H, generator=g) * 3, (torch.randn(T, H, generator=g) * 0.02).to(dtype)
    wp, wn = torch.rand(H, generator=g) + 0.5, torch.rand(H, generator=g) + 0.5
    c = lambda t: t.to(device)
    for use_y, nxt in ((True, True), (True, False), (False, True)):
        x, a = ops.branch_norm(c(res), c(y) if use_y else None, c(wp) if use_y else None, c(wn) if nxt else None, 1e-3, dtype)
        want = res.double().numpy()
        if use_y:
            want = want + plain.rms_norm(y.double().numpy(), wp.double().numpy(), 1e-3)
        assert x.dtype == torch.float32 and rel(x, want) < 1e-6
        if nxt:
            assert a.dtype == dtype and rel(a, plain.rms_norm(want, wn.double().numpy(), 1e-3)) < (3e-3 if dtype == torch.bfloat16 else 1e-6)
        else:
            assert a is None


# --------------------------------------------------------------------------- attention
def rope_state(spec, device):
    r = spec.rotary
    return RopeState(opref.rope_inv_freq(r.dims, r.base, r.scaling, device=device, dtype=torch.float64), r.pairing,
                     opref.rope_mscale(r.scaling), 0, 1, r.dims, 4096)


def batch(lens, page, device, seed=0, slots=None):
    """(meta, pages): rows fed and context lengths of every sequence, on shuffled pages; ``host_lens`` included."""
    g = torch.Generator().manual_seed(seed)
    nb = [(c + page - 1) // page for _, c in lens]
    perm = torch.randperm(sum(nb) + 2, generator=g).int()
    bt, o = torch.zeros(len(lens), max(nb), dtype=torch.int32), 0
    for b, k in enumerate(nb):
        bt[b, :k] = perm[o : o + k]
        o += k
    pos = torch.cat([torch.arange(c - n, c) for n, c in lens]).int()
    seq = torch.repeat_interleave(torch.arange(len(lens)), torch.tensor([n for n, _ in lens]))
    sl = (bt[seq, (pos // page).long()] * page + pos % page).int()
    qs = torch.tensor([0] + list(itertools.accumulate(n for n, _ in lens)), dtype=torch.int32)
    c = lambda t: t.to(device)
    return BatchMeta(None, c(pos), c(sl), c(qs), c(torch.tensor([x for _, x in lens], dtype=torch.int32)), c(bt), None,
                     max(n for n, _ in lens), max(x for _, x in lens), len(lens), host_lens=list(lens),
                     state_slots=None if slots is None else c(torch.tensor(slots, dtype=torch.int32))), sum(nb) + 2


def attention_plain(z, qn, kn, spec, sink, eps=1e-5):
    """Whole sequence from its unpadded projections z [T, q | k | v]; [T, heads, v_dim]."""
    T, H, G, d, vd = z.shape[0], spec.heads, spec.kv_heads, spec.dim, spec.v_dim
    q, k, v = z[:, : H * d], z[:, H * d : (H + G) * d], z[:, (H + G) * d :].reshape(T, G, vd)
    if spec.qk_norm == "full":
        q, k = plain.rms_norm(q, qn, eps), plain.rms_norm(k, kn, eps)
    q, k = q.reshape(T, H, d), k.reshape(T, G, d)
    if spec.qk_norm == "head":
        q, k = plain.rms_norm(q, qn, eps), plain.rms_norm(k, kn, eps)
    rot = {"dims": spec.rotary.dims, "base": spec.rotary.base}
    q, k = plain.rotate_heads(q, rot), plain.rotate_heads(k, rot)
    out = np.zeros((T, H, vd))
    for i in range(T):
        seen = list(plain.visible(i, spec.window if spec.window > 0 else i + 1))
        for h in range(H):
            s = k[seen, h // (H // G)] @ q[i, h] * spec.scale
            out[i, h] = plain.softmax(s, None if sink is None else float(sink[h])) @ v[seen, h // (H // G)]
    return out


def pad_rows(z, spec):
    """Unpadded projections as the kernels take them."""
    H, G, d, vd, W = spec.heads, spec.kv_heads, spec.dim, spec.v_dim, spec.width
    q, k, v = z[:, : H * d], z[:, H * d : (H + G) * d], z[:, (H + G) * d :]
    return torch.cat([pad_heads(q, H, W, 1), pad_heads(k, G, W, 1), pad_heads(v, G, W, 1)], 1).contiguous()


def pad_norms(qn, kn, spec):
    if not spec.qk_norm:
        return None, None
    full = spec.qk_norm == "full"
    return (pad_heads(qn, spec.heads if full else 1, spec.width).float().contiguous(),
            pad_heads(kn, spec.kv_heads if full else 1, spec.width).float().contiguous())


def run_attention(zs, qn, kn, spec, sink, lens, page, device, dtype, scale=1.0, splits=None, prefill_rows=None):
    """Every sequence's first rows go into the cache in a step of their own, then ``lens`` is one step; its outputs, unpadded."""
    eps = 1e-5
    meta, pages = batch(lens, page, device)
    kv = KVCache(KVCacheSpec(1, spec.kv_heads, spec.width, page, "bf16" if dtype == torch.bfloat16 else "f32"), pages, device)
    kv.data[0].fill_(3.0)  # nothing may rest on rows that were not written
    rope, (qw, kw) = rope_state(spec, device), pad_norms(qn, kn, spec)
    c = lambda t: None if t is None else t.to(device)
    qw, kw, sk = c(qw), c(kw), c(sink)
    past = [(x - n, x - n) for n, x in lens]
    rows = lambda which: pad_rows(torch.cat([z[lo:hi] for z, (lo, hi) in zip(zs, which)]), spec).to(device, dtype)
    if device == "cpu":
        prep, C = opref.head_prep, None
    else:
        from oxidize_b200.ops import cuda as C, cuda_latent as CLat, cuda_listed as CL

        prep = CL.head_prep
    if sum(n for n, _ in past):
        pm, _ = batch([p for p in past], page, device)
        slots = []
        for b, (n, _) in enumerate(past):
            p = torch.arange(n)
            slots.append((meta.block_tables[b].cpu()[p // page] * page + p % page).int())
        pm.slot_mapping = torch.cat(slots).to(device)
        prep(rows([(0, n) for n, _ in past]), qw, kw, spec, rope, pm, kv, 0, eps)
    q = prep(rows([(x - n, x) for n, x in lens]), qw, kw, spec, rope, meta, kv, 0, eps)
    T = q.shape[0]
    if device == "cpu":
        out = opref.paged_attention(q, kv, 0, meta, spec.scale, spec.window, sink=sk).reshape(T, -1) * scale
    else:
        wide = torch.full((T, spec.out_dim + 32), 9.0, dtype=dtype, device=device)
        out = wide[:, : spec.out_dim]
        if splits is not None:
            C.paged_attention(q, kv, 0, meta, spec.scale, spec.window, splits=splits, sink=sk, out=out, out_scale=scale)
        else:
            old, CLat.EXPAND_ROWS = CLat.EXPAND_ROWS, prefill_rows or CLat.EXPAND_ROWS
            try:
                CL.attention(q, kv, 0, meta, spec, sk, out, scale)
            finally:
                CLat.EXPAND_ROWS = old
        assert bool((wide[:, spec.out_dim :] == 9.0).all())
    out = out.reshape(T, spec.heads, spec.width)
    if spec.v_dim < spec.width:
        assert float(out[..., spec.v_dim :].abs().max()) == 0
    return out[..., : spec.v_dim]


CASES = [  # heads, kv heads, dim, v dim, rotated, window, norm, sink, (rows, context) per sequence, page
    (6, 2, 24, 20, 8, 19, "head", False, [(1, 100), (1, 5), (1, 19)], 16), (6, 2, 24, 20, 8, 19, "full", True, [(37, 100), (1, 5), (2, 64)], 16),
    (4, 4, 64, 64, 64, 0, "head", True, [(1, 300), (4, 130)], 16), (8, 1, 128, 128, 32, 130, "full", True, [(1, 400), (1, 131)], 16),
    (2, 1, 2, 1, 2, 1, "head", True, [(9, 20), (64, 64)], 8), (5, 5, 96, 80, 22, 65, "", False, [(3, 128), (2, 65)], 16),
    (3, 1, 192, 130, 64, 50, "full", True, [(2, 260), (1, 33)], 16), (4, 2, 256, 256, 256, 64, "head", False, [(20, 70)], 16),
    (2, 2, 300, 290, 100, 33, "head", True, [(3, 70)], 16), (6, 3, 40, 48, 40, 33, "full", True, [(150, 150)], 32),
    (7, 7, 32, 32, 6, 77, "full", True, [(64, 200), (1, 90), (300, 300), (2, 33), (70, 71)], 16),
    (4, 2, 128, 96, 128, 100, "head", True, [(257, 500)], 16), (12, 2, 64, 64, 16, 0, "head", False, [(200, 333), (65, 65)], 16)]


def case_of(c, seed=0):
    H, G, d, vd, rot, window, norm, sk, lens, page = c
    g = torch.Generator().manual_seed(seed + H * 100 + d)
    spec = AttentionSpec(H, G, d, vd, 2.5 / d ** 0.5, RotarySpec(rot, 1e4), window, sk, norm)
    zs = [torch.randn(x, (H + G) * d + G * vd, generator=g).bfloat16().float() for _, x in lens]
    n = (H * d, G * d) if norm == "full" else (d, d)
    qn, kn = torch.rand(n[0], generator=g) + 0.5, torch.rand(n[1], generator=g) + 0.5
    sink = torch.randn(H, generator=g) * 2 if sk else None
    return spec, zs, qn, kn, sink, lens, page


def attention_want(zs, qn, kn, spec, sink, lens):
    w = [attention_plain(z.double().numpy(), qn.double().numpy(), kn.double().numpy(), spec, None if sink is None else sink.double().numpy())
         for z in zs]
    return torch.tensor(np.concatenate([o[x - n : x] for o, (n, x) in zip(w, lens)]))


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("case", CASES, ids=str)
def test_attention_over_paged_rows(case, device, dtype):
    spec, zs, qn, kn, sink, lens, page = case_of(case)
    want = attention_want(zs, qn, kn, spec, sink, lens) * 0.75
    got = run_attention(zs, qn, kn, spec, sink, lens, page, device, dtype, 0.75)
    assert worst_row(got.reshape(got.shape[0], -1), want.reshape(got.shape[0], -1)) < (0.03 if dtype == torch.bfloat16 else 1e-5)


@gpu
@pytest.mark.parametrize("splits", [1, 3, 16])
def test_attention_key_splits_count_the_sink_once(splits):
    spec, zs, qn, kn, sink, lens, page = case_of((8, 2, 64, 64, 32, 300, "head", True, [(1, 420), (3, 300), (1, 2)], 16))
    got = run_attention(zs, qn, kn, spec, sink, lens, page, "cuda", torch.bfloat16, splits=splits)
    want = attention_want(zs, qn, kn, spec, sink, lens)
    assert worst_row(got.reshape(5, -1), want.reshape(5, -1)) < 0.03


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("rows", [1, 8, 100])
@pytest.mark.parametrize("window", [1, 2, 15, 16, 17, 48, 63, 64, 65, 130])
def test_window_edges_and_page_borders(device, dtype, rows, window):
    """One key stands out (its score is far above all others, and its value is its position's own): the query at distance
    window - 1 takes it all, the next one nothing of it.  The key sits on every place of a page in turn."""
    d = 32
    spec = AttentionSpec(2, 1, d, d, 8.0, RotarySpec(2, 1e9), window, False, "head")
    for key in (160, 167, 175, 191):
        ctx = key + window + 1
        z = torch.zeros(ctx, 4 * d)
        z[:, 4], z[:, d + 4] = 1.0, 1.0  # both heads' queries point along value 4 (past the rotated ones)
        z[:, 2 * d + 5] = 1.0
        z[key, 2 * d + 5], z[key, 2 * d + 4] = 0.0, 1.0
        z[:, 3 * d] = 1.0
        z[key, 3 * d : 3 * d + 2] = torch.tensor([0.0, 1.0])
        n = min(rows, ctx)
        out = run_attention([z], torch.ones(d), torch.ones(d), spec, None, [(n, ctx)], 16, device, dtype).float().cpu()
        inside, outside = out[-2, 0] if n > 1 else None, out[-1, 0]
        assert float(outside[1]) < 1e-3, (key, "the key just outside the window was seen")
        if n > 1:
            assert float(inside[1]) > 0.999, (key, "the key just inside the window was missed")
            if window > 1:
                last_in = min(n - 1, window)  # the farthest row of this step that sees the key
                assert float(out[-last_in, 0, 1]) > 0.999


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
def test_sink_takes_its_share_from_the_first_token_on(device, dtype):
    """Equal scores of zero: n visible keys and a sink s leave n / (n + exp(s)) of the value, also where n is 1."""
    spec = AttentionSpec(2, 2, 32, 32, 1.0, RotarySpec(2, 1e4), 3, True, "head")
    sink = torch.tensor([1.5, -30.0])
    z = torch.zeros(70, 6 * 32)
    z[:, 4 * 32 :] = 1.0
    for lens in ([(70, 70)], [(1, 1)], [(2, 70)]):
        out = run_attention([z[: lens[0][1]]], torch.ones(32), torch.ones(32), spec, sink, lens, 16, device, dtype).float().cpu()
        n = torch.tensor([min(p + 1, 3) for p in range(lens[0][1] - lens[0][0], lens[0][1])]).float()
        assert torch.allclose(out[:, 0, 0], n / (n + np.exp(1.5)), atol=4e-3) and torch.allclose(out[:, 1, 0], torch.ones_like(n), atol=4e-3)


@gpu
@pytest.mark.parametrize("case", [c for c in CASES if max(n for n, _ in c[8]) >= 64 and c[9] == 16], ids=str)
def test_long_portions_agree_with_the_paged_kernel(case):
    spec, zs, qn, kn, sink, lens, page = case_of(case)
    a = run_attention(zs, qn, kn, spec, sink, lens, page, "cuda", torch.bfloat16, prefill_rows=32)
    b = run_attention(zs, qn, kn, spec, sink, lens, page, "cuda", torch.bfloat16, prefill_rows=1 << 30)
    assert worst_row(a.reshape(a.shape[0], -1), b.double().cpu().reshape(a.shape[0], -1)) < 0.03


# --------------------------------------------------------------------------- retention
def retention_case(H, d, vd, rot, decay, lens, seed=0):
    g = torch.Generator().manual_seed(seed + d)
    spec = RetentionSpec(H, d, vd, list(decay), RotarySpec(rot, 1e4))
    zs = [torch.randn(x, 2 * H * (d + vd), generator=g).bfloat16().float() for _, x in lens]
    return spec, zs


def retention_want(z, spec, eps=1e-5):
    T, H, d, vd = z.shape[0], spec.heads, spec.dim, spec.v_dim
    rot = {"dims": spec.rotary.dims, "base": spec.rotary.base}
    q = plain.rotate_heads(z[:, : H * d].reshape(T, H, d), rot)
    k = plain.rotate_heads(z[:, H * d : 2 * H * d].reshape(T, H, d), rot) * d ** -0.5
    v, g = z[:, 2 * H * d : 2 * H * d + H * vd].reshape(T, H, vd), z[:, 2 * H * d + H * vd :]
    o = np.stack([plain.retention_scan(q[:, h], k[:, h], v[:, h], spec.decay[h]) for h in range(H)], axis=1)
    return plain.unit_rms(o, eps).reshape(T, H * vd) * plain.silu(g)


def ret_rows(z, spec):
    H, d, vd = spec.heads, spec.dim, spec.v_dim
    cut = [H * d, 2 * H * d, 2 * H * d + H * vd]
    parts = (z[:, : cut[0]], z[:, cut[0] : cut[1]], z[:, cut[1] : cut[2]], z[:, cut[2] :])
    return torch.cat([pad_heads(p, H, w, 1) for p, w in zip(parts, (spec.k_width, spec.k_width, spec.v_width, spec.v_width))], 1).contiguous()


def run_retention(z, spec, lens, slots, state, device, dtype, scale=1.0, **kw):
    meta, _ = batch(lens, 16, device, slots=slots)
    rope = rope_state(spec, device)
    z = ret_rows(z, spec).to(device, dtype)
    if device == "cpu":
        out = opref.retention(z, spec, rope, meta, state, 1e-5) * scale
    else:
        from oxidize_b200.ops import cuda_listed as CL

        wide = torch.full((z.shape[0], spec.out_dim + 16), 9.0, dtype=dtype, device=device)
        out = wide[:, : spec.out_dim]
        CL.retention(z, spec, rope, meta, state, torch.tensor(spec.decay, dtype=torch.float32, device=device), 1e-5, out, scale, **kw)
        assert bool((wide[:, spec.out_dim :] == 9.0).all())
    out = out.reshape(z.shape[0], spec.heads, spec.v_width)
    if spec.v_dim < spec.v_width:
        assert float(out[..., spec.v_dim :].abs().max()) == 0
    return out[..., : spec.v_dim].reshape(z.shape[0], -1)


RET = [  # heads, dim, v dim, rotated, decays
    (3, 24, 20, 16, [0.9, 0.97, 1.0]), (2, 64, 64, 64, [0.999, 0.5]), (1, 128, 128, 128, [0.9995]), (2, 96, 112, 6, [0.99, 0.7]),
    (1, 2, 1, 2, [0.75]), (4, 160, 48, 32, [0.98, 0.9, 0.6, 0.9999]), (2, 256, 250, 64, [0.97, 0.999])]


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("case", RET, ids=str)
@pytest.mark.parametrize("cuts", [[200], [1], [2, 3], [64], [63, 65], [9, 1, 8], [100, 2], [130, 70]], ids=str)
def test_retention_however_it_is_cut(case, cuts, device, dtype):
    """Steps and chunks in any order carry the state on; every row against the plain scan."""
    H, d, vd, rot, decay = case
    n = 200 if (device != "cpu" or cuts == [200]) else 40
    spec, (z,) = retention_case(H, d, vd, rot, decay, [(n, n)])
    state = torch.randn(3, *spec.state_shape, device=device)
    keep, out, at, i = state.clone(), [], 0, 0
    while at < n:
        m = min(cuts[i % len(cuts)], n - at)
        out.append(run_retention(z[at : at + m], spec, [(m, at + m)], [1], state, device, dtype, 0.5))
        at, i = at + m, i + 1
    want = retention_want(z.double().numpy(), spec) * 0.5
    err = worst_row(torch.cat(out), want)  # (a head of one value is divided by its own magnitude: rounding near zero grows)
    assert err < (0.02 if dtype == torch.bfloat16 else 2e-5 if vd > 1 else 2e-3), err
    assert torch.equal(state[0], keep[0]) and torch.equal(state[2], keep[2])


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
def test_retention_of_unequal_sequences_in_one_step(device, dtype):
    """Single tokens, short and long portions and a row without a slot beside each other; slots in any order."""
    lens = [(1, 40), (70, 70), (3, 100), (1, 1), (9, 9), (1, 1), (130, 200), (2, 2)]
    spec, zs = retention_case(2, 64, 48, 32, [0.99, 0.9], lens)
    slots = [5, 2, 7, 0, 1, -1, 3, 6]
    state = torch.full((8, *spec.state_shape), 11.0, device=device)
    for b, (n, x) in enumerate(lens):
        if x > n:
            run_retention(zs[b][: x - n], spec, [(x - n, x - n)], [slots[b]], state, device, dtype)
    got = run_retention(torch.cat([z[x - n :] for z, (n, x) in zip(zs, lens)]), spec, lens, slots, state, device, dtype)
    o = 0
    for b, (n, x) in enumerate(lens):
        want = retention_want(zs[b].double().numpy(), spec)[x - n :]
        if slots[b] < 0:
            assert float(got[o : o + n].abs().max()) == 0
        else:
            assert worst_row(got[o : o + n], want) < (0.02 if dtype == torch.bfloat16 else 2e-5), b
        o += n
    assert bool((state[4] == 11.0).all())


@gpu
@pytest.mark.parametrize("K,V", [(128, 128), (64, 96), (32, 16), (192, 64)])
@pytest.mark.parametrize("n_seg", [1, 2, 5])
@pytest.mark.parametrize("form", [1, 2])
def test_retention_segments_and_their_state(K, V, n_seg, form):
    """A long portion in segments leaves the same outputs and, to float32 rounding of split products, the same state as the
    float32 steps; with a decay of one nothing is forgotten over the whole length."""
    if form == 2 and K > 128:
        return
    lens = [(500, 700), (321, 321), (64, 128), (1, 7)]
    spec, zs = retention_case(2, K, V, 16, [1.0, 0.995], lens, seed=n_seg)
    z = torch.cat([x[c - n :] for x, (n, c) in zip(zs, lens)])
    first = torch.randn(4, *spec.state_shape, device="cuda")
    a, b = first.clone(), first.clone()
    want = run_retention(z, spec, lens, [3, 1, 0, 2], a, "cuda", torch.float32)
    got = run_retention(z, spec, lens, [3, 1, 0, 2], b, "cuda", torch.bfloat16, n_seg=n_seg, form=form)
    assert worst_row(got, want.double().cpu()) < 0.02
    for s in range(4):
        assert rel(b[s], a[s]) < 3e-5, s


@gpu
@pytest.mark.parametrize("form", [1, 2])
def test_retention_keeps_32_bits_of_what_enters_the_recurrence(form):
    """One early key and value, and a query far behind that stands on it: with a decay of one the output before the norm is
    their product; factors rounded to 16 bits would show in the state."""
    spec = RetentionSpec(1, 64, 64, [1.0], RotarySpec(64, 1e4))
    g = torch.Generator().manual_seed(3)
    z = torch.zeros(600, 256)
    z[3] = torch.randn(256, generator=g).bfloat16().float()
    state = torch.zeros(1, 1, 64, 64, device="cuda")
    run_retention(z, spec, [(600, 600)], [0], state, "cuda", torch.bfloat16, n_seg=3, form=form)
    k = plain.rotate_heads(np.pad(z[3:4, None, 64:128].double().numpy(), ((3, 0), (0, 0), (0, 0))), {"dims": 64, "base": 1e4})[3, 0] / 8
    want = np.outer(k, z[3, 128:192].double().numpy())
    assert rel(state[0, 0], want) < 2e-5


# --------------------------------------------------------------------------- feed-forward blocks
def ffn_weights(H, F, g):
    return [(torch.randn(n, k, generator=g) / k ** 0.5).bfloat16().float() for n, k in ((F, H), (F, H), (H, F))]


def np_ffn(x, gate, up, down):
    x, gate, up, down = (t.double().numpy() for t in (x, gate, up, down))
    return (plain.silu(x @ gate.T) * (x @ up.T)) @ down.T


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("T,H,F", [(1, 64, 64), (7, 40, 1), (65, 96, 88), (130, 256, 512), (3, 42, 10)])
def test_gated_feed_forward(device, dtype, T, H, F):
    from oxidize_b200.models.config import ModelConfig

    g = torch.Generator().manual_seed(F)
    ws, x = ffn_weights(H, F, g), torch.randn(T, H, generator=g).bfloat16().float()
    spec = FeedForwardSpec(F, "silu", True)
    gu, down = gated_pair(*[w.to(device, dtype) for w in ws], spec.pad_size)
    gu, down = LinearWeight([gu]), LinearWeight([down])
    if dtype == torch.bfloat16:
        from oxidize_b200.ops import cuda as C

        gu.parts[0].data, gu.swiglu_interleaved = C.interleave_gate_up(gu.parts[0].data), True
    got = ops.gated_ffn(x.to(device, dtype), gu, down)
    assert rel(got, np_ffn(x, *ws)) < (1e-2 if dtype == torch.bfloat16 else 1e-6)


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("T,H,E,top,F,shared", [(1, 64, 8, 2, 32, 48), (5, 42, 3, 3, 10, None), (200, 128, 16, 4, 64, 1), (64, 96, 1, 1, 5, 7),
                                                (300, 64, 60, 6, 24, None), (9, 256, 256, 8, 8, 64)])
def test_routed_experts(device, dtype, T, H, E, top, F, shared):
    g = torch.Generator().manual_seed(E + T)
    spec = MoESpec(E, top, FeedForwardSpec(F, "silu", True), FeedForwardSpec(shared, "silu", True) if shared else None)
    x = torch.randn(T, H, generator=g).bfloat16().float()
    router = (torch.randn(E, H, generator=g) * 2 / H ** 0.5).bfloat16().float()
    experts = [ffn_weights(H, F, g) for _ in range(E)]
    sh = ffn_weights(H, shared, g) if shared else None
    c = lambda t: t.to(device, dtype)
    lw = LayerWeights(attn_norm=None, wqkv=None, wo=None, ffn_norm=None,
                      router=QTensor("F32" if dtype == torch.float32 else "BF16", c(router), (E, H)),
                      experts=listed_experts(spec, [[c(w) for w in e] for e in experts], H))
    if sh:
        gu, down = gated_pair(*[c(w) for w in sh], spec.shared.pad_size)
        lw.shared_gate_up, lw.shared_down = LinearWeight([gu]), LinearWeight([down])
    got = ops.moe_ffn(c(x), lw, spec)
    z = x.double().numpy() @ router.double().numpy().T
    want = np.zeros((T, H))
    for t in range(T):
        for e, w in zip(*plain.choose(z[t], top)):
            want[t] += w * np_ffn(x[t : t + 1], *experts[e])[0]
    if sh:
        want += np_ffn(x, *sh)
    assert got.dtype == dtype and worst_row(got, want) < (0.03 if dtype == torch.bfloat16 else 1e-5)


@gpu
@pytest.mark.parametrize("T,E,K", [(1, 8, 16), (17, 30, 4096), (64, 64, 1000), (2048, 60, 2048), (3, 5, 42)])
def test_router_logits_are_not_rounded(T, E, K):
    """bf16 operands, float32 sums: far closer to the exact product than a 16-bit result could be."""
    from oxidize_b200.ops import cuda_listed as CL

    g = torch.Generator().manual_seed(K)
    x, w = torch.randn(T, K, generator=g).bfloat16(), torch.randn(E, K, generator=g).bfloat16()
    got = CL.router_logits(x.cuda(), QTensor("BF16", w.cuda(), (E, K)))
    assert got.dtype == torch.float32 and rel(got, x.double() @ w.double().T) < 2e-6


# --------------------------------------------------------------------------- states, configuration, what is refused
def test_state_slots_are_handed_out_once():
    s = StateSlots(3)
    a = [s.allocate() for _ in range(3)]
    assert sorted(a) == [0, 1, 2]
    with pytest.raises(OutOfBlocks):
        s.allocate()
    s.release(a[1])
    with pytest.raises(RuntimeError):
        s.release(a[1])
    assert s.allocate() == a[1]


def small(**over):
    rot = plain.rotation
    cfg = plain.config(32, 40, [(plain.attn(4, 2, 8, 8, 9, rot(4)), plain.dense(24)),
                                (plain.parallel(plain.attn(2, 1, 8, 8, 12, rot(8)), plain.ret(2, 8, 8, [0.9, 0.8], rot(8)), 1.0, 0.5),
                                 plain.moe(4, 2, 8)), 0])
    cfg.update(over)
    return cfg


def test_reader_and_parameter_count(tmp_path):
    from oxidize_b200.formats.layered import open_checkpoint
    from oxidize_b200.models.registry import config_from_checkpoint

    cfg = small()
    w = plain.random_weights(cfg)
    mc = config_from_checkpoint(open_checkpoint(plain.write_model(str(tmp_path / "m"), cfg, w)))
    assert mc.arch == "sokirax" and mc.norm_placement == "sandwich" and mc.has_state and not mc.is_ssm
    assert mc.param_count() == sum(t.size for t in w.values())
    assert mc.uniform_window == 12 and len(mc.cache_shapes) == 3 and mc.state_shapes == [(2, 32, 16)]
    a, p, c = mc.layer_specs
    assert isinstance(p.mixer, ParallelSpec) and p.branch_scales == (1.0, 0.5) and p.mixer.left.qk_norm == "full" and p.mixer.left.sink
    assert a.mixer.qk_norm == "head" and not a.mixer.sink and c.weights_of == 0 and c.mixer == a.mixer
    assert isinstance(p.ffn, MoESpec) and p.ffn.shared is None and a.ffn.gated


def bad(change):
    cfg = small()
    change(cfg["layers"])
    return cfg


@pytest.mark.parametrize("cfg", [
    bad(lambda l: l[0].update(type="convolution")), bad(lambda l: l[2].update(weights_of=2)), bad(lambda l: l[2].update(weights_of=1)),
    bad(lambda l: l[2].update(weights_of=7)), bad(lambda l: l[0]["mlp"].update(kind="other")), bad(lambda l: l[0]["mixer"].update(kv_heads=3)),
    bad(lambda l: l[1]["mixer"]["right"].update(decay=[0.5])), bad(lambda l: l[1]["mixer"]["right"].update(decay=[0.5, 1.5])),
    bad(lambda l: l[1]["mlp"]["router"].update(top=9)), bad(lambda l: l[0]["mixer"]["rot"].update(dims=10))], ids=str)
def test_configurations_that_are_refused(tmp_path, cfg):
    from oxidize_b200.formats.layered import open_checkpoint
    from oxidize_b200.models.registry import config_from_checkpoint

    path = plain.write_model(str(tmp_path / "m"), small(), plain.random_weights(small()))
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    with pytest.raises((ValueError, UnsupportedArchitecture)):
        config_from_checkpoint(open_checkpoint(path))


def test_what_such_a_model_cannot_do_is_refused(tmp_path):
    from oxidize_b200.engine.spec import attach_speculation
    from oxidize_b200.formats.layered import open_checkpoint
    from oxidize_b200.models.registry import config_from_checkpoint, load_checkpoint_weights

    path = plain.write_model(str(tmp_path / "m"), small(), plain.random_weights(small()))
    ck = open_checkpoint(path)
    with pytest.raises(ValueError, match="sharded"):
        load_checkpoint_weights(ck, config_from_checkpoint(ck), tp_size=2)
    llm = LLM.from_checkpoint(path, EngineConfig(max_model_len=32, max_num_seqs=2), device="cpu")
    with pytest.raises(ValueError, match="rolled back"):
        attach_speculation(llm, path)
    assert llm.kv.states.nbytes() == 2 * 2 * 32 * 16 * 4


def test_a_layer_may_be_retention_alone():
    """The mixers are parts: a listed layer with a state and no attention owns no cache rows."""
    from oxidize_b200.models.layered import layered_config
    from oxidize_b200.models.transformer import Transformer
    from oxidize_b200.utils.synth import synth_weights

    r = RetentionSpec(2, 8, 8, [0.9, 0.8], RotarySpec(8, 1e4))
    a = AttentionSpec(2, 1, 8, 8, 0.3, RotarySpec(8, 1e4), 5)
    cfg = layered_config("listed", 30, 32, [LayerSpec(r, FeedForwardSpec(16, "silu", True)), LayerSpec(a, None), LayerSpec(r, None)], 1e-5,
                         "rms", norm_placement="sandwich")
    assert cfg.cache_shapes == [(1, 2, 32)] and len(cfg.state_shapes) == 2 and cfg.uniform_window == 5
    llm = LLM(synth_weights(cfg, "cpu", "F32", seed=1), EngineConfig(max_model_len=64, max_num_seqs=2))
    assert llm.model.kv_index == [-1, 0, -1] and llm.model.state_index == {0: 0, 2: 1}
    from oxidize_b200.engine.sampler import SamplingParams

    sp = SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True)
    one = [o.token_ids for o in llm.generate([[1, 2, 3]], sp)]
    assert one == [o.token_ids for o in llm.generate([[1, 2, 3]], sp)]
