"""The mechanisms behind models that list their layers, one at a time: norm after the sum, latent attention (window edges,
sink, page borders, key splits), rotation, rows taken from another layer, the products around them, configuration checks."""
import itertools
import math

import numpy as np
import pytest
import torch

import vefilix_plain as plain
from oxidize_b200 import ops
from oxidize_b200.engine.kv_pool import KVCache, KVCacheSpec
from oxidize_b200.engine.llm import LLM, EngineConfig
from oxidize_b200.models.config import LatentAttentionSpec, RotarySpec, UnsupportedArchitecture
from oxidize_b200.models.transformer import BatchMeta
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


# --------------------------------------------------------------------------- norms and products
@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("T,H", [(1, 4), (5, 96), (3, 257), (7, 4096), (2, 6144), (2, 10002)])
@pytest.mark.parametrize("kind", ["layer", "rms"])
def test_norm_after_the_sum(device, dtype, T, H, kind):
    g = torch.Generator().manual_seed(H)
    res, y = torch.randn(T, H, generator=g) * 3 + 5, (torch.randn(T, H, generator=g) * 2).to(dtype)
    w, b = torch.rand(H, generator=g) + 0.5, torch.randn(H, generator=g)
    for use_res, use_y, bias in ((True, True, True), (True, False, True), (False, True, False)):
        z = (2.5 * res.double().numpy() if use_res else 0) + (y.double().numpy() if use_y else 0)
        bb = b.double().numpy() if bias else 0.0
        want = plain.layer_norm(z, w.double().numpy(), bb, 1e-3) if kind == "layer" else plain.rms_norm(z, w.double().numpy(), 1e-3) + bb
        x, a = ops.residual_norm(res.to(device) if use_res else None, y.to(device) if use_y else None, 2.5, w.to(device),
                                 b.to(device) if bias else None, 1e-3, kind, dtype)
        assert x.dtype == torch.float32 and a.dtype == dtype
        assert rel(x, want) < 2e-6 and rel(a, want) < (1e-5 if dtype == torch.float32 else 4e-3)


@gpu
@pytest.mark.parametrize("T,N,K", [(1, 51, 40), (3, 7, 5), (130, 203, 96), (65, 64, 1000), (600, 520, 36)])
def test_products_in_32_bits_and_with_the_relu2_epilogue(T, N, K):
    from oxidize_b200.models.layered import dense_qtensor
    from oxidize_b200.models.weights import LinearWeight

    g = torch.Generator().manual_seed(T)
    x, w = torch.randn(T, K, generator=g).cuda(), (torch.randn(N, K, generator=g) / K ** 0.5).cuda()
    want = x.double() @ w.double().t()
    lin = LinearWeight([dense_qtensor(w)])
    assert rel(ops.linear(x, lin), want) < 1e-6  # no shortened operands (TF32 would give 3e-4)
    assert rel(ops.linear_act(x, lin, "relu2"), want.clamp(min=0) ** 2) < 2e-6
    xb, wb = x.bfloat16(), w.bfloat16()
    want = xb.double() @ wb.double().t()
    lin = LinearWeight([dense_qtensor(wb)])
    assert rel(ops.linear(xb, lin), want) < 5e-3
    assert rel(ops.linear_act(xb, lin, "relu2"), want.clamp(min=0) ** 2) < 5e-3


@gpu
@pytest.mark.parametrize("H,T,N,K", [(1, 1, 8, 8), (3, 5, 20, 16), (8, 300, 100, 24), (5, 70, 33, 136), (32, 64, 512, 128)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_products_per_head(H, T, N, K, dtype):
    from oxidize_b200.ops import cuda_latent as CL

    x, w = torch.randn(H, T, K, device="cuda").to(dtype), torch.randn(H, N, K, device="cuda").to(dtype)
    y = torch.zeros(T, H * N + 8, dtype=dtype, device="cuda")
    CL.batched(x, w, y, N, H * N + 8)
    want = torch.einsum("htk,hnk->thn", x.double(), w.double()).reshape(T, H * N)
    assert rel(y[:, : H * N], want) < (1e-6 if dtype == torch.float32 else 5e-3) and not y[:, H * N :].any()


# --------------------------------------------------------------------------- rotation
@pytest.mark.parametrize("dims,base,s", [(16, 1e4, None), (12, 5e5, dict(factor=8.0, original=128, fast=32.0, slow=1.0)),
                                         (8, 1e6, dict(factor=2.0, original=4096, fast=4.0, slow=0.001)),
                                         (2, 1e4, dict(factor=1.0, original=64, fast=8.0, slow=1.0)),
                                         (6, 3e4, dict(factor=0.5, original=64, fast=8.0, slow=1.0))])
def test_rotation_frequencies(dims, base, s):
    """The ramp's end may lie past the last pair; cos and sin carry the magnitude for every factor."""
    from oxidize_b200.models.layered import _yarn

    f, mag = plain.frequencies({"dims": dims, "base": base, "scaling": s})
    sc = _yarn(s, dims)
    assert np.allclose(opref.rope_inv_freq(dims, base, sc, dtype=torch.float64).numpy(), f, rtol=1e-12)
    assert math.isclose(opref.rope_mscale(sc), mag, rel_tol=1e-12)
    x = torch.randn(3, 2, dims + 4)
    got = opref.apply_rope(x, torch.tensor([0, 7, 1000]), opref.rope_inv_freq(dims, base, sc, dtype=torch.float64), "split_half",
                           opref.rope_mscale(sc))
    for i, p in enumerate((0, 7, 1000)):
        assert rel(got[i, 1], plain.rotate(x[i, 1].double().numpy(), p, {"dims": dims, "base": base, "scaling": s})) < 1e-6


# --------------------------------------------------------------------------- attention over cached rows
def rows_setup(ctx, rank, rot, page, device, dtype, seed=0):
    """A cache with shuffled pages for sequences of the given lengths; returns (cache, block tables, rows per sequence)."""
    g = torch.Generator().manual_seed(seed)
    spec = LatentAttentionSpec(1, 8, rot, 8, rank, 1.0, RotarySpec(rot, 1e4))
    nb = [(n + page - 1) // page for n in ctx]
    kv = KVCache(KVCacheSpec(1, 1, spec.row_dim, page, "bf16" if dtype == torch.bfloat16 else "f32", planes=1), sum(nb) + 2, device)
    order = torch.randperm(sum(nb) + 2, generator=g).tolist()
    bt, rows, o = torch.zeros(len(ctx), max(nb), dtype=torch.int32), [], 0
    for b, n in enumerate(ctx):
        bt[b, : nb[b]] = torch.tensor(order[o : o + nb[b]])
        o += nb[b]
        r = torch.randn(n, spec.row_dim, generator=g).to(dtype).float()
        r[:, rank : spec.latent_pad] = 0
        r[:, spec.latent_pad + rot :] = 0
        rows.append(r)
    return spec, kv, bt, rows, g


def put_rows(kv, bt, rows, page):
    for b, r in enumerate(rows):
        slots = torch.tensor([int(bt[b, p // page]) * page + p % page for p in range(r.shape[0])], dtype=torch.int32)
        opref.kv_write(kv, 0, r[:, None].to(kv.data[0].device), None, slots.to(kv.data[0].device))


def attend(q, kv, bt, qlens, ctx, spec, sink, device, dtype, splits=None, plain_kernel=False):
    """[T, H, rank] through the path of the device; q [T, H, row]."""
    qs = torch.tensor([0] + list(itertools.accumulate(qlens)), dtype=torch.int32, device=device)
    meta = BatchMeta(None, None, None, qs, torch.tensor(ctx, dtype=torch.int32, device=device), bt.to(device), None, max(qlens), max(ctx),
                     len(ctx))
    q = q.to(device, dtype)
    sk = None if sink is None else sink.to(device)
    if device == "cpu":
        return opref.latent_attention(q, kv, 0, meta, spec.scale, spec.kv_rank, spec.window, sk)
    from oxidize_b200.ops import cuda_latent as CL

    out = torch.full((q.shape[1], q.shape[0], spec.latent_pad), 7.0, dtype=dtype, device=device)
    if dtype == torch.float32 or plain_kernel:
        CL.attention_simt(q, kv, 0, meta, spec, sk, out)
    else:
        assert CL.attention_mma(q, kv, 0, meta, spec, sk, out, splits)
        again = torch.full_like(out, 3.0)
        CL.attention_mma(q, kv, 0, meta, spec, sk, again, splits)
        assert torch.equal(out, again)  # reproducible, and nothing but the output written
    return out.permute(1, 0, 2)[..., : spec.kv_rank]


def attend_plain(q, rows, qlens, ctx, spec, sink):
    out, t = [], 0
    for b, n in enumerate(qlens):
        k = rows[b].double().numpy()
        for i in range(ctx[b] - n, ctx[b]):
            seen = list(plain.visible(i, spec.window)) if spec.window > 0 else list(range(i + 1))
            for h in range(q.shape[1]):
                s = k[seen] @ q[t, h].double().numpy() * spec.scale
                p = plain.softmax_with_sink(s, float(sink[h]) if sink is not None else -1e30)
                out.append(p @ k[seen][:, : spec.kv_rank])
            t += 1
    return torch.tensor(np.array(out)).reshape(q.shape[0], q.shape[1], -1)


CASES = [  # heads, rank, rotated, window, rows per sequence, context lengths, page, key splits
    (5, 40, 6, 19, [1, 1, 1], [100, 5, 19], 16, None), (5, 40, 6, 19, [37, 1, 2], [100, 5, 64], 16, 1),
    (3, 96, 8, 0, [1, 4], [300, 130], 16, 3), (12, 136, 24, 130, [1, 1], [400, 131], 32, 2), (2, 24, 2, 1, [9, 1], [20, 64], 8, None),
    (40, 200, 16, 65, [3, 2], [128, 65], 64, None), (7, 512, 64, 100, [2, 1], [260, 33], 16, 2), (33, 64, 64, 64, [70], [70], 16, None),
    (4, 48, 8, 0, [1], [1500], 16, 12), (4, 48, 8, 0, [1], [300], 16, 16)]


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("case", CASES, ids=str)
def test_attention_over_cached_rows(case, device, dtype):
    H, rank, rot, window, qlens, ctx, page, splits = case
    spec, kv, bt, rows, g = rows_setup(ctx, rank, rot, page, device, dtype)
    spec.heads, spec.window, spec.scale = H, window, 2.0 / spec.row_dim ** 0.5
    put_rows(kv, bt, rows, page)
    q = torch.randn(sum(qlens), H, spec.row_dim, generator=g).to(dtype).float()
    for sink in (torch.randn(H, generator=g) + 2, None):
        want = attend_plain(q, rows, qlens, ctx, spec, sink)
        tol = 1e-5 if dtype == torch.float32 else 6e-3
        assert rel(attend(q, kv, bt, qlens, ctx, spec, sink, device, dtype, splits), want) < tol
        if dtype == torch.bfloat16:
            assert rel(attend(q, kv, bt, qlens, ctx, spec, sink, device, dtype, plain_kernel=True), want) < tol


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("page", [8, 16])
@pytest.mark.parametrize("window", [1, 16, 17, 63, 64, 65, 130])
def test_window_edges_and_page_borders(window, page, device, dtype):
    """One key stands out for every query.  While it is inside the window the output is its value; one position later it
    contributes nothing.  In a portion of several rows and one row at a time, around every page border."""
    n = 200
    spec, kv, bt, rows, g = rows_setup([n], 16, 2, page, device, dtype, seed=window)
    spec.window, spec.scale, spec.heads = window, 1.0, 2
    q = torch.zeros(1, 2, spec.row_dim)
    q[..., 0] = 1.0
    for far in (0, page - 1, page, 3 * page - 1, 63, 64):
        r = rows[0].clone()
        r[:, 0] = 0.0
        r[far, 0] = 30.0  # a score of 30 against 0
        put_rows(kv, bt, [r], page)
        first = max(far - 1, 0)
        last = min(far + window + 1, n - 1)  # far + window - 1 is the last position that sees the key
        m = last - first + 1
        got = [attend(q.expand(m, -1, -1).clone(), kv, bt, [m], [last + 1], spec, None, device, dtype)]  # one portion
        got.append(torch.cat([attend(q, kv, bt, [1], [p + 1], spec, None, device, dtype)
                              for p in {first, far, far + window - 1, far + window} if p <= last]))
        at = [list(range(first, last + 1)), [p for p in {first, far, far + window - 1, far + window} if p <= last]]
        for out, where in zip(got, at):
            for o, p in zip(out.float().cpu(), where):
                inside = far <= p < far + window
                near = float((o[:, 1:] - r[far, 1:16]).abs().max())
                assert (near < 0.05) == inside, (far, p)
                if not inside:
                    assert float(o[:, 0].abs().max()) < 1e-6  # not a trace of it


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
def test_sink_joins_the_denominator_once(device, dtype):
    """Equal scores of n keys and a sink of log(n): the output is half the mean value, however the keys are split."""
    for n, splits in ((1, 1), (7, 1), (128, 2), (400, 4), (400, 1)):
        spec, kv, bt, rows, _ = rows_setup([n], 16, 2, 16, device, dtype, seed=n)
        spec.scale, spec.window, spec.heads = 1.0, 0, 3
        put_rows(kv, bt, rows, 16)
        sink = torch.tensor([math.log(n), -1e4, math.log(n) + 40.0])
        o = attend(torch.zeros(1, 3, spec.row_dim), kv, bt, [1], [n], spec, sink, device, dtype, splits).float().cpu()[0]
        mean = rows[0][:, :16].mean(0)
        tol = 1e-6 if dtype == torch.float32 else 1e-2
        assert torch.allclose(o[0], mean / 2, atol=tol) and torch.allclose(o[1], mean, atol=tol) and float(o[2].abs().max()) < 1e-6


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
def test_scores_that_grow_along_the_keys(device, dtype):
    """Every tile raises the running maximum by far more than the lazy margin of the kernel, and very negative scores."""
    n = 500
    spec, kv, bt, rows, g = rows_setup([n], 32, 2, 16, device, dtype)
    spec.scale, spec.window, spec.heads = 1.0, 0, 2
    q = torch.zeros(3, 2, spec.row_dim)
    q[..., 0], q[:, 1, 0] = 1.0, -1.0
    rows[0][:, 0] = (torch.arange(n) * 0.5).to(dtype).float()
    put_rows(kv, bt, rows, 16)
    sink = torch.tensor([3.0, -200.0])
    want = attend_plain(q, rows, [3], [n], spec, sink)
    assert rel(attend(q, kv, bt, [3], [n], spec, sink, device, dtype, 2), want) < (1e-5 if dtype == torch.float32 else 6e-3)


# --------------------------------------------------------------------------- configuration, loading, sharding
def test_configurations_that_are_refused(tmp_path):
    base = [(plain.mixer(2, 8, 4, 8, 16, 9), 16), (plain.mixer(2, 8, 4, 8, 16, 9, kv_from=0), 16)]

    def load(change, layers=base):
        cfg = plain.config(32, 40, [(dict(m, rot=dict(m["rot"])), f) for m, f in layers])
        w = plain.random_weights(cfg)
        change(cfg)
        path = plain.write_model(str(tmp_path / "m"), cfg, w)
        return LLM.from_checkpoint(path, EngineConfig(max_model_len=32, num_kv_blocks=8, max_num_seqs=2), device="cpu")

    assert load(lambda c: None).cfg.uniform_window == 9
    for change, err in [(lambda c: c.update(architecture="Other"), UnsupportedArchitecture),
                        (lambda c: c["layers"][0].update(type="attention"), UnsupportedArchitecture),
                        (lambda c: c["layers"][1]["mlp"].update(kind="gated"), UnsupportedArchitecture),
                        (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=2), UnsupportedArchitecture),
                        (lambda c: c["layers"][1]["mixer"].update(kv_from=1), ValueError),
                        (lambda c: c["layers"][1]["mixer"].update(kv_rank=8), ValueError),
                        (lambda c: c["layers"][1]["mixer"]["rot"].update(base=5.0), ValueError)]:
        with pytest.raises(err):
            load(change)


def test_cache_holds_one_row_per_owning_layer(tmp_path):
    cfg = plain.config(32, 40, [(plain.mixer(2, 8, 4, 8, 16, 9), 16), (plain.mixer(2, 8, 4, 8, 16, 5, kv_from=0), 16),
                                (plain.mixer(2, 8, 6, 8, 40, 12), None)])
    llm = LLM.from_checkpoint(plain.write_model(str(tmp_path / "m"), cfg, plain.random_weights(cfg)),
                              EngineConfig(max_model_len=32, num_kv_blocks=8, max_num_seqs=2), device="cpu")
    assert [tuple(d.shape) for d in llm.kv.data] == [(8, 1, 1, 16, 32), (8, 1, 1, 16, 64)]
    assert llm.model.kv_index == [0, 0, 1] and llm.kv.spec.bytes_per_block() == (32 + 64) * 16 * 4
    state = llm.kv.state_dict([1, 2])
    llm.kv.load_state_dict(state, [3, 4])


def test_heads_and_feed_forward_are_sharded_over_ranks(tmp_path):
    """Two ranks' outputs add up to the single rank's (what the all-reduce does), layer by layer inputs being equal."""
    from oxidize_b200.formats.layered import open_checkpoint
    from oxidize_b200.models.registry import config_from_checkpoint, load_checkpoint_weights
    from oxidize_b200.models.transformer import Transformer

    cfg = plain.config(32, 40, [(plain.mixer(4, 8, 4, 6, 16, 9), 24)])
    ck = open_checkpoint(plain.write_model(str(tmp_path / "m"), cfg, plain.random_weights(cfg)))
    mc = config_from_checkpoint(ck)
    x = torch.randn(20, 32)
    i32 = dict(dtype=torch.int32)
    pos = torch.arange(20, **i32)
    meta = BatchMeta(pos, pos, pos, torch.tensor([0, 20], **i32), torch.tensor([20], **i32), torch.tensor([[0, 1]], **i32), None, 20, 20, 1)

    def branch(rank, size):
        w = load_checkpoint_weights(ck, mc, tp_rank=rank, tp_size=size)
        lw, spec = w.layers[0], mc.layer_specs[0]
        kv = KVCache(KVCacheSpec(1, 1, 32, 16, "f32", planes=1, shapes=((1, 1, 32),)), 2, "cpu")
        rope = Transformer(load_checkpoint_weights(ck, mc), max_context=64).layer_ropes[0][0]
        a = ops.linear(ops.latent_mixer(x, lw.mla, spec.mixer, rope, meta, kv, 0, mc.rms_eps), lw.wo)
        return a, ops.linear(ops.linear_act(x, lw.w_up, "relu2"), lw.w_down)

    whole, parts = branch(0, 1), [branch(r, 2) for r in range(2)]
    for i in range(2):
        assert rel(parts[0][i] + parts[1][i], whole[i]) < 1e-6


# --------------------------------------------------------------------------- the whole mixer on the device, both forms
MIXERS = [  # heads, nope, rot, v, rank, window, (rows, context) per sequence, page
    (3, 24, 8, 20, 40, 19, [(100, 100)], 16), (4, 128, 64, 128, 512, 130, [(300, 700), (64, 64), (257, 300)], 16),
    (2, 16, 16, 16, 48, 1, [(65, 65)], 8), (5, 40, 6, 36, 72, 64, [(1, 200), (1, 3), (128, 128), (70, 400), (2, 90)], 16),
    (2, 64, 32, 96, 128, 0, [(200, 513)], 32), (1, 192, 16, 8, 32, 77, [(90, 150), (64, 65)], 64), (2, 8, 2, 1, 16, 500, [(64, 64)], 16)]


@gpu
@pytest.mark.parametrize("case", MIXERS, ids=str)
def test_expanded_and_absorbed_forms_agree_with_the_32_bit_path(case, monkeypatch):
    """Long portions attend over expanded keys and values, short ones over the cached rows; in one step beside each other.
    Every row against the float32 path on the same (16-bit representable) inputs, with attention peaked on single keys."""
    from oxidize_b200.models.layered import latent_weights
    from oxidize_b200.models.transformer import RopeState
    from oxidize_b200.ops import cuda_latent as CL

    H, nope, rot, v, rank, window, lens, page = case
    g = torch.Generator().manual_seed(H * 100 + v)
    rnd = lambda *s: torch.randn(*s, generator=g).bfloat16().float()
    spec = LatentAttentionSpec(H, nope, rot, v, rank, 3.0 / (nope + rot) ** 0.5, RotarySpec(rot, 1e4), window, True)
    T, W = sum(n for n, _ in lens), H * (nope + rot) + rank + rot
    qkv = rnd(T, W)
    uk, uv = rnd(H * nope, rank) / rank ** 0.5, rnd(H * v, rank) / rank ** 0.5
    norm, sink = torch.rand(rank, generator=g) + 0.5, torch.randn(H, generator=g)
    nb = [(c + page - 1) // page for _, c in lens]
    perm = torch.randperm(sum(nb), generator=g).int()
    bt = torch.zeros(len(lens), max(nb), dtype=torch.int32)
    o = 0
    for b, k in enumerate(nb):
        bt[b, :k] = perm[o : o + k]
        o += k
    past = rnd(sum(nb), 1, 1, page, spec.row_dim)
    past[..., rank : spec.latent_pad] = 0
    past[..., spec.latent_pad + rot :] = 0
    pos = torch.cat([torch.arange(c - n, c) for n, c in lens]).int()
    seq = torch.repeat_interleave(torch.arange(len(lens)), torch.tensor([n for n, _ in lens]))
    slots = (bt[seq, (pos // page).long()] * page + pos % page).int()
    qs = torch.tensor([0] + list(itertools.accumulate(n for n, _ in lens)), dtype=torch.int32)

    def run(dtype, expand):
        monkeypatch.setattr(CL, "EXPAND_ROWS", expand)
        c = lambda t: t.cuda()
        m = latent_weights(spec, torch.zeros(H * (nope + rot), 8), torch.zeros(rank + rot, 8), c(norm), c(uk.to(dtype)), c(uv.to(dtype)),
                           c(sink))
        kv = KVCache(KVCacheSpec(1, 1, spec.row_dim, page, "bf16" if dtype == torch.bfloat16 else "f32", planes=1), sum(nb), "cuda")
        kv.data[0].copy_(past)
        meta = BatchMeta(None, c(pos), c(slots), c(qs), c(torch.tensor([x for _, x in lens], dtype=torch.int32)), c(bt), None,
                         max(n for n, _ in lens), max(x for _, x in lens), len(lens), host_lens=list(lens))
        rope = RopeState(opref.rope_inv_freq(rot, 1e4, None, device="cuda", dtype=torch.float64), "split_half", 1.0, 0, 1, rot, 1024)
        out = CL.latent_core(c(qkv).to(dtype), m, spec, rope, meta, kv, 0, 1e-5, CL.operands(m, spec, dtype))
        return out.double().cpu(), kv.data[0].double().cpu()

    want, rows = run(torch.float32, 1 << 30)
    scale = float(want.pow(2).mean().sqrt())
    for expand in (64, 1 << 30):  # the second: everything in absorbed form
        got, r16 = run(torch.bfloat16, expand)
        assert rel(r16, rows) < 4e-3
        err = (got - want).pow(2).mean(-1).sqrt() / scale
        assert float(err.max()) < 0.08 and float(err.mean()) < 0.02, (expand, float(err.max()), int(err.argmax()), float(err.mean()))
