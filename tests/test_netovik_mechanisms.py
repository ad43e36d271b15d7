"""The mechanisms of layers with norms on their branches' outputs, one at a time: grouped norm with sum and depth average, token
shift, decays, RWKV time mixing (steps, chunks, portions, state slots), attention on the scores of all heads together (windows
with kept first tokens, distance buckets, mixing, soft cap, the extra one in the denominator, key splits, long portions), routed
experts with plain scores, pages of kept first tokens, configuration checks."""
import dataclasses
import json
import os

import numpy as np
import pytest
import torch

import netovik_plain as plain
from oxidize_b200 import ops
from oxidize_b200.engine.kv_pool import BlockPool, KVCache, KVCacheSpec, StateStore
from oxidize_b200.engine.llm import LLM, EngineConfig
from oxidize_b200.engine.sampler import SamplingParams
from oxidize_b200.engine.scheduler import Scheduler, SchedulerConfig, Sequence
from oxidize_b200.models.config import AttentionSpec, FeedForwardSpec, MoESpec, UnsupportedArchitecture, WkvSpec, distance_bucket
from oxidize_b200.models.layered import distance_bias, distance_rows, listed_experts, pad_heads, wkv_weights
from oxidize_b200.models.weights import LayerWeights, QTensor
from oxidize_b200.ops import ref as opref
from test_listed_mixers import B16, CPU, F32, batch, gpu, rel, worst_row

TOL = {torch.float32: 2e-5, torch.bfloat16: 1.5e-2}


@pytest.fixture(autouse=True)
def _status():
    yield
    if torch.cuda.is_available():
        from oxidize_b200.ops import cuda as C

        assert C.status()[0] == 0


# --------------------------------------------------------------------------- norm, sum, depth average
@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("T,H,groups", [(1, 4, 1), (5, 96, 3), (3, 257, 1), (7, 4096, 2), (2, 6144, 8), (600, 2048, 4), (2, 10002, 6),
                                        (3, 64, 64), (4, 384, 3), (3, 200, 20), (2, 16384, 1)])
def test_grouped_norm_joins_the_stream(device, dtype, T, H, groups):
    g = torch.Generator().manual_seed(H + T)
    res, y = torch.randn(T, H, generator=g) * 3, torch.randn(T, H, generator=g)
    y.view(T, groups, -1).mul_(torch.logspace(-3, 2, groups)[None, :, None])  # (parts of very different size)
    y, w = y.to(dtype), torch.rand(H, generator=g) + 0.5
    k = 3
    rows = torch.randn(T * k, H + 4, generator=g).to(dtype)  # routed rows may be wider than the model
    index, share = torch.randperm(T * k, generator=g).reshape(T, k).int(), torch.rand(T, k, generator=g)
    c, n = lambda t: t.to(device), lambda t: t.double().numpy()
    ys = [(c(y), n(y))]
    if device != "cpu":
        ys.append((ops.RoutedRows(c(rows), c(index), c(share)), (n(rows)[index.numpy(), :H] * n(share)[:, :, None]).sum(1)))
    for branch, want in ys:
        want = n(res) + plain.grouped_norm(want, n(w), groups, 1e-3)
        for act in (dtype, None):
            x, a = ops.add_normed(c(res), branch, c(w), groups, 1e-3, act)
            assert x.dtype == torch.float32 and rel(x, want) < 1e-6
            assert (a is None) if act is None else a.dtype == act and rel(a, want) < (3e-3 if dtype == torch.bfloat16 else 1e-6)
    a = ops.grouped_norm(c(res), c(w), groups, 1e-3, dtype)
    assert a.dtype == dtype and rel(a, plain.grouped_norm(n(res), n(w), groups, 1e-3)) < (3e-3 if dtype == torch.bfloat16 else 1e-6)


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("T,H,groups", [(3, 96, 3), (5, 1024, 2), (1, 42, 1)])
def test_depth_average_weighs_every_result_so_far(device, dtype, T, H, groups):
    """Twelve layers; each result is kept as it is ahead of the average that goes on."""
    g = torch.Generator().manual_seed(H)
    c, n = lambda t: t.to(device), lambda t: t.double().numpy()
    x = torch.randn(T, H, generator=g)
    streams = ops.DepthStreams(c(x), 12)
    results, now, dev = [n(x)], n(x), c(x)
    for i in range(12):
        y, w, depth = torch.randn(T, H, generator=g).to(dtype), torch.rand(H, generator=g) + 0.5, torch.randn(i + 2, generator=g)
        results.append(now + plain.grouped_norm(n(y), n(w), groups, 1e-5))
        now = plain.depth_average(results, n(depth))
        dev, a = ops.add_normed(dev, c(y), c(w), groups, 1e-5, dtype, streams, c(depth))
        assert rel(dev, now) < 2e-6 and rel(a, now) < (3e-3 if dtype == torch.bfloat16 else 2e-6)
        assert rel(streams.results[i], results[-1]) < 2e-6 and streams.n == i + 1


# --------------------------------------------------------------------------- token shift and decays
def mixer_case(H, d, rank, hidden, dtype, seed=0, decay=-2.0, spread=1.5):
    """(spec, tensors as a checkpoint stores them)."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    t = {n: r(H * d, hidden) / hidden ** 0.5 for n in "rkvg"}
    t.update({"w1": r(rank, hidden) / hidden ** 0.5, "w2": r(H * d, rank) / rank ** 0.5, "o": r(hidden, H * d) / (H * d) ** 0.5})
    t = {n: x.bfloat16().to(dtype) for n, x in t.items()}
    t.update({"mu." + n: 0.5 + 0.3 * r(hidden) for n in "rkvgw"})
    t.update({"w0": spread * r(H * d) + decay, "u": r(H, d), "norm": 1 + 0.2 * r(H * d)})
    return WkvSpec(H, d, rank, hidden), t


def to_device(w, device):
    for f in ("mu", "proj", "decay_up", "decay_base", "bonus", "norm"):
        setattr(w, f, getattr(w, f).to(device))
    for p in w.decay_down.parts:
        p.data = p.data.to(device)
    return w


class MixerRun:
    """Sequences fed portion by portion through the whole mixer, each with its own slot."""

    def __init__(self, spec, t, device, dtype, slots=6):
        self.spec, self.device, self.dtype = spec, device, dtype
        self.w = to_device(wkv_weights(spec, t, dtype)["wkv"], device)
        self.store = StateStore([spec.state_shape], slots, device, [spec.window_shape])
        self.store.data[0].fill_(7.0)  # nothing of an earlier owner may be seen
        self.store.windows[0].fill_(-5.0)

    def step(self, parts):
        """``parts``: (input rows, rows before them, slot); outputs of all rows, unpadded."""
        x = torch.cat([x for x, _, _ in parts]).to(self.device)
        meta, _ = batch([(len(x), past + len(x)) for x, past, _ in parts], 16, self.device, slots=[s for _, _, s in parts])
        out = ops.wkv_mixer(x, self.w, self.spec, meta, self.store.data[0], self.store.windows[0], 1e-5, self.dtype)
        out = out.reshape(-1, self.spec.heads, self.spec.v_width)
        assert not out[..., self.spec.dim :].any()
        return out[..., : self.spec.dim]

    def feed(self, x, cuts, slot=2):
        out, at = [], 0
        for n in cuts:
            out.append(self.step([(x[at : at + n], at, slot)]))
            at += n
        assert at == len(x)
        return torch.cat(out)


def mixer_plain(spec, t, x, eps=1e-5):
    """(outputs [T, heads, dim] ahead of the output projection, final states)."""
    H, d, T = spec.heads, spec.dim, len(x)
    n = {k: v.double().numpy() for k, v in t.items()}
    at = {s: plain.shifted(x, n["mu." + s]) for s in "rkvgw"}
    r, k, v = ((at[s] @ n[s].T).reshape(T, H, d) for s in "rkv")
    dec = plain.decays(at["w"], n["w1"], n["w2"], n["w0"]).reshape(T, H, d)
    heads = [plain.wkv_scan(r[:, h], k[:, h], v[:, h], dec[:, h], n["u"][h]) for h in range(H)]
    o = plain.unit_rms(np.stack([a for a, _ in heads], 1), eps) * n["norm"].reshape(H, d)
    return o * plain.silu(at["g"] @ n["g"].T).reshape(T, H, d), np.stack([s for _, s in heads])


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("hidden", [8, 42, 96, 1030, 4096])
def test_token_shift_across_portions(device, dtype, hidden):
    """The row ahead of a portion's first comes from the step before, in a batch of portions and single tokens, on slots that
    held something else; a padding row leaves nothing behind."""
    g = torch.Generator().manual_seed(hidden)
    mu = torch.rand(3, hidden, generator=g).to(device)
    xs = [torch.randn(n, hidden, generator=g) for n in (9, 4, 6)]
    wants = [np.stack([plain.shifted(x.double().numpy(), m) for m in mu.double().cpu().numpy()]) for x in xs]
    window = torch.full((5, 1, hidden), 11.0, device=device)
    slots, at = [3, 0, 4], [0, 0, 0]
    for sizes in ([4, 1, 0], [1, 2, 3], [2, 1, 2], [1, 0, 1], [1, 0, 0]):
        rows = [(i, n) for i, n in enumerate(sizes) if n] + [(1, 1)]
        ids = [slots[i] for i, _ in rows[:-1]] + [-1]
        x = torch.cat([xs[i][at[i] : at[i] + n] if s >= 0 else xs[1][:1] for (i, n), s in zip(rows, ids)]).to(device)
        meta, _ = batch([(n, (at[i] if s >= 0 else 0) + n) for (i, n), s in zip(rows, ids)], 16, device, slots=ids)
        if device == "cpu":
            got = opref.token_shift(x, mu, meta, window)
        else:
            from oxidize_b200.ops import cuda_wkv

            got = cuda_wkv.token_shift(x, mu, meta, window, dtype)
            assert not got[..., hidden:].any()
            got = got[..., :hidden]
        o = 0
        for i, n in rows[:-1]:
            assert rel(got[:, o : o + n], wants[i][:, at[i] : at[i] + n]) < (4e-3 if dtype == torch.bfloat16 else 1e-6)
            at[i] += n
            o += n
            assert torch.equal(window[slots[i], 0].cpu(), xs[i][at[i] - 1])
    assert at == [9, 4, 6] and (window[[1, 2]] == 11.0).all()


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("H,d,rank,hidden", [(2, 24, 5, 40), (3, 64, 32, 64), (1, 1, 1, 8), (4, 128, 100, 128), (2, 32, 700, 48)])
def test_decays_from_their_two_projections(device, dtype, H, d, rank, hidden):
    spec, t = mixer_case(H, d, rank, hidden, dtype)
    w = to_device(wkv_weights(spec, t, dtype)["wkv"], device)
    low = torch.randn(37, rank, generator=torch.Generator().manual_seed(1)).to(dtype) * 2
    padded = torch.nn.functional.pad(low, (0, spec.decay_dim - rank)).to(device)
    if device == "cpu":
        got = opref.wkv_log_decay(padded, w)
    else:
        from oxidize_b200.ops import cuda_wkv

        got = cuda_wkv.log_decay(padded, w)
    got = got.reshape(37, H, spec.k_width)[..., :d].reshape(37, H * d)
    z = low.double().numpy()
    want = np.log(plain.decays(z, np.eye(rank), t["w2"].double().numpy(), t["w0"].double().numpy()))
    assert got.dtype == torch.float32 and rel(got, want) < 1e-5


# --------------------------------------------------------------------------- RWKV time mixing
WKV_SHAPES = [(2, 24, 5, 40), (4, 64, 16, 96), (1, 3, 1, 8), (3, 128, 40, 64), (2, 96, 7, 70), (5, 33, 3, 42), (2, 160, 8, 64), (1, 250, 8, 32)]


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("shape", WKV_SHAPES, ids=str)
def test_time_mixing_however_a_sequence_is_cut(device, dtype, shape):
    """Whole, token by token, in portions that end anywhere in a chunk: outputs, the final state and the last input."""
    spec, t = mixer_case(*shape, dtype)
    T = 150
    x = torch.randn(T, spec.hidden, generator=torch.Generator().manual_seed(1))
    want, state = mixer_plain(spec, t, x.double().numpy())
    for cuts in ([T], [1] * T, [2, 3] * 30, [1, 64, 1, 63, 21], [100, 1, 1, 48], [9, 8] * 8 + [14]):
        run = MixerRun(spec, t, device, dtype)
        got = run.feed(x, cuts)
        err = worst_row(got.flatten(1), want.reshape(T, -1))
        assert err < (8e-2 if dtype == torch.bfloat16 else 1e-4), (cuts, err)
        assert rel(got, want) < (1.5e-2 if dtype == torch.bfloat16 else 1e-5)
        assert rel(run.store.data[0][2][:, : spec.dim, : spec.dim], state) < (1e-2 if dtype == torch.bfloat16 else 1e-5), cuts
        assert torch.equal(run.store.windows[0][2, 0].cpu(), x[-1])
        assert (run.store.data[0][3] == 7.0).all() and (run.store.windows[0][3] == -5.0).all()


class ScanRun:
    """The recurrence alone on given projections and decays, one sequence in slot 1."""

    def __init__(self, H, d, device, dtype, seed=0, **kw):
        self.spec, t = mixer_case(H, d, 1, 8, dtype, seed)
        self.w, self.device, self.dtype, self.kw = to_device(wkv_weights(self.spec, t, dtype)["wkv"], device), device, dtype, kw
        self.u, self.norm = t["u"].double().numpy(), t["norm"].double().numpy().reshape(H, d)
        self.state = torch.full((3,) + self.spec.state_shape, 3.0, device=device)

    def feed(self, z, log_decay, cuts):
        """z [4, T, H * d] unpadded, log_decay [T, H * d]."""
        s, out, at = self.spec, [], 0
        zp = torch.stack([pad_heads(p, s.heads, s.k_width, 1) for p in z]).to(self.device, self.dtype)
        lp = pad_heads(log_decay.float(), s.heads, s.k_width, 1).to(self.device)
        for n in cuts:
            meta, _ = batch([(n, at + n)], 16, self.device, slots=[1])
            part, dec = zp[:, at : at + n], lp[at : at + n].contiguous()
            if self.device == "cpu":
                o = opref.wkv(part, dec, self.w, s, meta, self.state, 1e-5)
            else:
                from oxidize_b200.ops import cuda_wkv

                flat = part.transpose(0, 1).reshape(n, -1).contiguous()
                o = torch.full((n, s.out_dim), float("nan"), dtype=self.dtype, device=self.device)
                cuda_wkv.wkv(flat, dec, self.w, s, meta, self.state, 1e-5, o, **self.kw)
            out.append(o.reshape(n, s.heads, s.v_width)[..., : s.dim])
            at += n
        return torch.cat(out)

    def plain(self, z, log_decay):
        H, d = self.spec.heads, self.spec.dim
        r, k, v, g = z.double().numpy().reshape(4, -1, H, d)
        w = np.exp(log_decay.double().numpy()).reshape(-1, H, d)
        heads = [plain.wkv_scan(r[:, h], k[:, h], v[:, h], w[:, h], self.u[h]) for h in range(H)]
        return plain.unit_rms(np.stack([a for a, _ in heads], 1), 1e-5) * self.norm * plain.silu(g), np.stack([s for _, s in heads])


STATE_TOL = {torch.float32: 1e-5, torch.bfloat16: 4e-5}


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("d", [32, 40, 128])
def test_decays_of_every_strength(device, dtype, d):
    """Channels and tokens that forget (nearly) everything, others that forget nothing, and runs of both, at any place of a
    chunk: no exponent may overflow, and what lies behind a forgetting token stays exact."""
    T, H = 200, 2
    g = torch.Generator().manual_seed(2)
    z = torch.randn(4, T, H * d, generator=g).to(dtype).float()
    log_decay = -torch.exp(3.0 * torch.randn(T, H * d, generator=g) - 2.0)
    log_decay[torch.randperm(T, generator=g)[:20]] *= 100.0
    log_decay[70:90] = -1e-4
    log_decay[[3, 47, 48, 63, 64, 130]] = -300.0
    log_decay[:, 1] = -4.0  # (a whole block loses more than its range on one channel)
    log_decay[:, 5] = 0.0
    for cuts in ([T], [1] * T, [65, 65, 70], [9, 100, 91]):
        run = ScanRun(H, d, device, dtype)
        want, state = run.plain(z, log_decay)
        got = run.feed(z, log_decay, cuts)
        assert torch.isfinite(got.float()).all() and worst_row(got, want) < 2 * TOL[dtype], cuts
        assert rel(run.state[1][:, :d, :d], state) < STATE_TOL[dtype], cuts
        assert (run.state[[0, 2]] == 3.0).all()


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
def test_far_writes_are_remembered_and_the_bonus_is_the_current_tokens_alone(device, dtype):
    """No decay along one channel: one value written under that channel is read 300 tokens later; and a token whose own key
    answers its query through the bonus only."""
    T, d = 330, 64
    g = torch.Generator().manual_seed(3)
    z = 0.1 * torch.randn(4, T, d, generator=g)
    log_decay = torch.full((T, d), -0.5)
    log_decay[:, 7] = 0.0
    z[1, :, 7] = 0.0
    z[0, 320], z[1, 17], z[2, 17] = 0.0, 0.0, 3.0
    z[0, 320, 7], z[1, 17, 7] = 9.0, 9.0
    z[0, 200], z[1, 200], z[2, 200] = 0.0, 0.0, -4.0
    z[0, 200, 11], z[1, 200, 11] = 20.0, 20.0
    z = z.to(dtype).float()
    run = ScanRun(1, d, device, dtype)
    want, _ = run.plain(z, log_decay)
    hidden = z.clone()
    hidden[2, 17] = -3.0
    assert worst_row(want[320], run.plain(hidden, log_decay)[0][320]) > 0.5  # (the read-out hangs on that write)
    for cuts in ([T], [18, 1, 200, 101, 10], [300] + [1] * 30, [17, 183, 1, 129]):
        got = ScanRun(1, d, device, dtype).feed(z, log_decay, cuts)
        for t in (200, 320):
            assert worst_row(got[t], want[t]) < TOL[dtype], (cuts, t)
        assert worst_row(got, want) < 3 * TOL[dtype], cuts


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
def test_time_mixing_in_batches_and_on_reused_slots(device, dtype):
    """Long and short portions and single tokens of several sequences in one step, a padding row without a slot, and slots
    that a new sequence takes over."""
    spec, t = mixer_case(4, 64, 16, 48, dtype)
    g = torch.Generator().manual_seed(6)
    xs = [torch.randn(n, 48, generator=g) for n in (170, 12, 40, 75)]
    wants = [mixer_plain(spec, t, x.double().numpy())[0] for x in xs]
    run = MixerRun(spec, t, device, dtype)
    plan = [[(0, 0, 70), (1, 0, 1), (2, 0, 33)], [(2, 33, 34), (0, 70, 71), (1, 1, 8)], [(1, 8, 9), (2, 34, 35), (0, 71, 72)],
            [(0, 72, 170), (2, 35, 40), (1, 9, 12)], [(3, 0, 75)]]
    slots = {0: 4, 1: 0, 2: 5, 3: 4}
    got = {i: [] for i in slots}
    for entries in plan:
        out = run.step([(xs[i][lo:hi], lo, slots[i]) for i, lo, hi in entries] + [(xs[1][:1], 0, -1)])
        o = 0
        for i, lo, hi in entries:
            got[i].append(out[o : o + hi - lo])
            o += hi - lo
        assert not out[o:].any()
    for i in slots:
        assert rel(torch.cat(got[i]), wants[i]) < (1.5e-2 if dtype == torch.bfloat16 else 1e-5), i


@gpu
@pytest.mark.parametrize("rounds", [1, 2, 100])
@pytest.mark.parametrize("H,d", [(2, 24), (3, 64), (1, 96), (5, 128), (2, 112)])
def test_chunks_agree_with_steps(H, d, rounds):
    """The tensor-core kernels, in rounds of any number of chunks, against the token-by-token one on the same 16-bit rows, and
    twice the same."""
    g = torch.Generator().manual_seed(d)
    z = torch.randn(4, 333, H * d, generator=g).bfloat16().float()
    log_decay = -torch.exp(1.5 * torch.randn(333, H * d, generator=g) - 2.0)
    for cuts in ([333], [64, 128, 141], [9, 55, 269]):
        runs = [ScanRun(H, d, "cuda", torch.bfloat16, chunk_rows=r, rounds=rounds) for r in (2, 2, 1 << 20)]
        outs = [r.feed(z, log_decay, cuts) for r in runs]
        assert torch.equal(outs[0], outs[1]) and torch.equal(runs[0].state, runs[1].state)
        assert rel(runs[0].state[1], runs[2].state[1]) < 3e-5 and worst_row(outs[0], outs[2].cpu()) < 1e-2


# --------------------------------------------------------------------------- attention on the scores of all heads
@pytest.mark.parametrize("rows,far", [(2, 2), (2, 900), (8, 40), (12, 13), (32, 128), (32, 120), (32, 256), (64, 33), (6, 1000)])
def test_distance_buckets(rows, far):
    table = distance_rows(rows, far)
    for n in range(3 * far + rows):
        assert plain.bucket(n, rows, far) == distance_bucket(n, rows, far) == (table[n] if n < len(table) else rows - 1), n
    assert list(table) == sorted(table) and table[-1] == rows - 1


def joint_spec(H, G, d, window=0, keep=0, scale=0.4, cap=9.0, rows=8, far=30):
    return AttentionSpec(H, G, d, d, scale, None, window, qk_norm="unit", bias=True, keep_first=keep, softcap=cap, bias_rows=rows, bias_max=far,
                         talk=True, unit_sink=True, shared_kv=True)


def joint_case(spec, seed=0, mix=1.0, bias=1.0):
    g = torch.Generator().manual_seed(seed)
    rel_t, talk = bias * torch.randn(spec.bias_rows, spec.heads, generator=g), mix * torch.randn(spec.heads, spec.heads, generator=g) / spec.heads ** 0.5
    return rel_t, talk + torch.eye(spec.heads)


def joint_plain(spec, z, rel_t, talk, eps=1e-5):
    """[T, heads, dim] of a whole sequence from its unpadded projections z [T, q | k]."""
    T, H, G, d = len(z), spec.heads, spec.kv_heads, spec.dim
    q, k = z[:, : H * d].reshape(T, H, d), z[:, H * d :].reshape(T, G, d)
    m = {"scale": spec.scale, "softcap": spec.softcap, "bias_max": spec.bias_max, "mask": {"size": spec.window, "keep_first": spec.keep_first}}
    return plain.mixed_attention(plain.unit_rms(q, eps), plain.unit_rms(k, eps), k, m, rel_t.double().numpy(), talk.double().numpy())


class JointRun:
    """Sequences fed portion by portion on pages of one cache."""

    def __init__(self, spec, rel_t, talk, device, dtype, lens, page=16, form=None, **kw):
        self.spec, self.device, self.dtype, self.page, self.form, self.kw = spec, device, dtype, page, form, kw
        self.mix = talk.float().contiguous().to(device)
        self.bias = distance_bias(rel_t, spec.bias_max, talk).to(device)
        self.sink = torch.zeros(spec.heads, device=device)
        full, pages = batch([(n, n) for n in lens], page, device)
        self.tables = full.block_tables
        G, planes, width = spec.cache_shape
        self.kv = KVCache(KVCacheSpec(1, G, width, page, "bf16" if dtype == torch.bfloat16 else "f32", planes=planes), pages, device)
        self.kv.data[0].fill_(3.0)  # nothing may rest on rows that were not written

    def step(self, parts):
        """``parts``: (sequence, unpadded rows, rows before them); outputs, unpadded."""
        s = self.spec
        meta, _ = batch([(len(z), past + len(z)) for _, z, past in parts], self.page, self.device)
        meta.block_tables = self.tables[[i for i, _, _ in parts]].contiguous()
        seq = torch.repeat_interleave(torch.arange(len(parts)), torch.tensor([len(z) for _, z, _ in parts])).to(self.device)
        pos = meta.positions.long()
        meta.slot_mapping = (meta.block_tables[seq, pos // self.page] * self.page + pos % self.page).int()
        z = torch.cat([z for _, z, _ in parts])
        zp = torch.cat([pad_heads(z[:, : s.heads * s.dim], s.heads, s.width, 1), pad_heads(z[:, s.heads * s.dim :], s.kv_heads, s.width, 1)], 1)
        zp = zp.to(self.device, self.dtype).contiguous()
        if self.device == "cpu":
            q = opref.joint_prep(zp, s, meta, self.kv, 0, 1e-5)
            return opref.joint_attention(q, self.kv, 0, meta, s, self.bias, self.mix, self.sink, 1e-5)[..., : s.dim]
        from oxidize_b200.ops import cuda_joint as CJ
        from oxidize_b200.ops import cuda_listed as CL

        q = CL.head_prep(zp, None, None, s, None, meta, self.kv, 0, 1e-5)
        out = torch.full((len(z), s.heads * s.width), float("nan"), dtype=self.dtype, device=self.device)
        f = {None: CJ.attention, "simt": CJ.attention_simt, "decode": CJ.attention_decode, "prefill": CJ.attention_prefill}[self.form]
        f(q, self.kv, 0, meta, s, self.bias, self.mix, self.sink, out, 1.0, **self.kw)
        return out.reshape(-1, s.heads, s.width)[..., : s.dim]

    def feed(self, z, cuts, seq=0):
        out, at = [], 0
        for n in cuts:
            out.append(self.step([(seq, z[at : at + n], at)]))
            at += n
        return torch.cat(out)


FORMS = [pytest.param("cpu", torch.float32, None, id="cpu"), pytest.param("cuda", torch.float32, None, id="gpu32", marks=gpu)] + [
    pytest.param("cuda", torch.bfloat16, f, id=f"gpu16-{f}", marks=gpu) for f in ("simt", "decode", "prefill")]
PREFILL = {"long_rows": 1}


def joint_run(spec, rel_t, talk, device, dtype, lens, form):
    return JointRun(spec, rel_t, talk, device, dtype, lens, form=form, **(PREFILL if form == "prefill" else {}))


@pytest.mark.parametrize("device,dtype,form", FORMS)
@pytest.mark.parametrize("H,G,d,window,keep", [(6, 2, 24, 30, 5), (5, 5, 16, 48, 16), (8, 4, 32, 17, 21), (1, 1, 2, 1, 1), (7, 1, 40, 0, 0),
                                               (16, 16, 64, 33, 40), (32, 8, 128, 64, 4), (20, 20, 96, 50, 1), (3, 3, 100, 0, 0), (32, 32, 32, 16, 0),
                                               (28, 4, 64, 100, 64)])
def test_scores_of_all_heads_in_every_form(device, dtype, form, H, G, d, window, keep):
    spec = joint_spec(H, G, d, window, keep)
    rel_t, talk = joint_case(spec, H)
    T = 150 if d < 100 else 110
    z = torch.randn(T, (H + G) * d, generator=torch.Generator().manual_seed(d)).to(dtype).float()
    want = joint_plain(spec, z.double().numpy(), rel_t, talk)
    for cuts in ([T], [1, 16, 33, 1, T - 51]) + (([3] * 10 + [1] * (T - 30),) if form != "prefill" else ()):
        got = joint_run(spec, rel_t, talk, device, dtype, [T], form).feed(z, cuts)
        assert torch.isfinite(got.float()).all()
        assert worst_row(got.flatten(1), want.reshape(T, -1)) < (2e-2 if dtype == torch.bfloat16 else 2e-5), cuts


def standing_out(spec, T, j, i, size=8.0):
    """Projections in which key j answers query i far better than any other does, and its value is large."""
    g = torch.Generator().manual_seed(T + j)
    z = 0.3 * torch.randn(T, (spec.heads + spec.kv_heads) * spec.dim, generator=g)
    d, H = spec.dim, spec.heads
    a = torch.randn(d, generator=g)
    z[j, H * d :] = (size * a).repeat(spec.kv_heads)
    z[i, : H * d] = a.repeat(H)
    return z


@pytest.mark.parametrize("device,dtype,form", FORMS)
@pytest.mark.parametrize("window,keep", [(16, 0), (17, 3), (31, 16), (32, 5), (40, 32), (64, 33), (1, 1), (2, 2), (0, 0)])
def test_edges_of_windows_and_kept_tokens(device, dtype, form, window, keep):
    """One key that stands out just inside and just outside the window, among the last kept first tokens and the next, at page
    and tile borders; read by a query of a portion and by a decoded one."""
    spec = joint_spec(4, 2, 32, window, keep, scale=1.5, cap=50.0)
    rel_t, talk = joint_case(spec, 1, mix=0.2, bias=0.3)
    T, i = 120, 101
    size = window or T
    places = {max(0, i - size), max(0, i - size + 1), max(0, keep - 1), keep, 0, 15, 16, 31, 32, i - 1, i, 95, 96}
    for j in sorted(p for p in places if p <= i):
        z = standing_out(spec, T, j, i).to(dtype).float()
        want = joint_plain(spec, z.double().numpy(), rel_t, talk)
        if plain.visible(i, j, size, keep):  # (the output hangs on that key)
            other = z.clone()
            other[j, spec.heads * spec.dim :] *= -1.0
            assert worst_row(want[i], joint_plain(spec, other.double().numpy(), rel_t, talk)[i]) > 0.3
        for cuts in ([T], [i, 1, T - i - 1], [i - 1, 2, T - i - 1]):
            got = joint_run(spec, rel_t, talk, device, dtype, [T], form).feed(z, cuts)
            assert worst_row(got[i].flatten(), want[i].reshape(-1)) < (2.5e-2 if dtype == torch.bfloat16 else 2e-5), (j, cuts)


@pytest.mark.parametrize("device,dtype,form", FORMS)
def test_distance_bias_mixing_cap_and_the_extra_one_show(device, dtype, form):
    """Each of them changes the result by far more than the tolerance, on keys at every distance, and large biases move whole
    tiles apart (weights of tiles whose maxima differ by hundreds)."""
    T = 140
    base = joint_spec(6, 3, 32, 100, 8, scale=0.5, cap=4.0, rows=16, far=90)
    rel_t, talk = joint_case(base, 3, mix=2.0, bias=2.0)
    z = torch.randn(T, 9 * 32, generator=torch.Generator().manual_seed(5)).to(dtype).float()
    zn = z.double().numpy()
    want = joint_plain(base, zn, rel_t, talk)
    for other in (joint_plain(base, zn, rel_t.flip(0), talk), joint_plain(base, zn, rel_t, talk.t()),
                  joint_plain(dataclasses.replace(base, softcap=40.0), zn, rel_t, talk)):
        assert rel(want, other) > 0.1
    for scale_bias, cap in ((1.0, 4.0), (60.0, 4.0), (0.0, 1.0)):
        spec = dataclasses.replace(base, softcap=cap)
        want = joint_plain(spec, zn, rel_t * scale_bias, talk)
        got = joint_run(spec, rel_t * scale_bias, talk, device, dtype, [T], form).feed(z, [100, 40])
        assert worst_row(got.flatten(1), want.reshape(T, -1)) < (2e-2 if dtype == torch.bfloat16 else 5e-5), (scale_bias, cap)
    low = rel_t - 25.0  # scores far below that of the extra one: next to nothing comes out
    want = joint_plain(base, zn, low, torch.eye(6))
    assert np.abs(want).max() < 1e-2
    got = joint_run(base, low, torch.eye(6), device, dtype, [T], form).feed(z, [T])
    assert worst_row(got.flatten(1), want.reshape(T, -1)) < (4e-2 if dtype == torch.bfloat16 else 2e-5)


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("page", [16, 8, 32, 4])
def test_unequal_sequences_in_one_batch(device, dtype, page):
    """Portions of some beside single tokens of others on shuffled pages, each against itself alone."""
    spec = joint_spec(6, 2, 48, 37, 6)
    rel_t, talk = joint_case(spec, 4)
    lens = [130, 3, 60, 18]
    g = torch.Generator().manual_seed(8)
    zs = [torch.randn(n, 8 * 48, generator=g).to(dtype).float() for n in lens]
    run = JointRun(spec, rel_t, talk, device, dtype, lens, page)
    plan = [[(2, 0, 17), (0, 0, 70), (1, 0, 1)], [(0, 70, 71), (1, 1, 2), (2, 17, 50), (3, 0, 18)], [(2, 50, 52), (1, 2, 3), (0, 71, 130)],
            [(2, 52, 60)]]
    got = {i: [] for i in range(4)}
    for entries in plan:
        out = run.step([(i, zs[i][lo:hi], lo) for i, lo, hi in entries])
        o = 0
        for i, lo, hi in entries:
            got[i].append(out[o : o + hi - lo])
            o += hi - lo
    for i, n in enumerate(lens):
        want = joint_plain(spec, zs[i].double().numpy(), rel_t, talk)
        assert worst_row(torch.cat(got[i]).flatten(1), want.reshape(n, -1)) < (2e-2 if dtype == torch.bfloat16 else 2e-5), i


@gpu
@pytest.mark.parametrize("splits", [1, 2, 3, 8, 16])
@pytest.mark.parametrize("H,G,d", [(32, 8, 128), (12, 12, 64), (4, 1, 32), (2, 2, 256), (6, 3, 192), (48, 4, 32)])
def test_key_splits_of_a_decoded_token(H, G, d, splits):
    """A long context dealt out to any number of CTAs, with and without a window; twice the same."""
    for window, keep in ((0, 0), (300, 20)):
        spec = joint_spec(H, G, d, window, keep, rows=32, far=128)
        rel_t, talk = joint_case(spec, 7)
        T = 700
        z = torch.randn(T, (H + G) * d, generator=torch.Generator().manual_seed(d)).bfloat16().float()
        one = lambda run: torch.cat([run.step([(0, z[t : t + 1], t)]) for t in range(T - 3, T)])
        slow = JointRun(spec, rel_t, talk, "cuda", torch.bfloat16, [T], form="simt")
        slow.feed(z[:-3], [T - 3])
        outs = []
        for _ in range(2):
            run = JointRun(spec, rel_t, talk, "cuda", torch.bfloat16, [T], form="decode", splits=splits)
            run.tables, run.kv = slow.tables, slow.kv
            outs.append(one(run))
        want = one(slow)
        assert torch.equal(outs[0], outs[1]) and worst_row(outs[0].flatten(1), want.flatten(1).cpu()) < 1e-2


@gpu
@pytest.mark.parametrize("H,G,d,window,keep", [(32, 8, 128, 200, 4), (32, 32, 64, 0, 0), (6, 6, 80, 128, 40), (17, 17, 32, 90, 7), (9, 3, 16, 50, 1)])
def test_long_portions_in_several_launches(H, G, d, window, keep):
    """Scratch for few blocks at a time, portions of two sequences behind what earlier steps left, against the plain kernel."""
    spec = joint_spec(H, G, d, window, keep, rows=32, far=128)
    rel_t, talk = joint_case(spec, 9)
    g = torch.Generator().manual_seed(d)
    lens = [600, 333]
    zs = [torch.randn(n, (H + G) * d, generator=g).bfloat16().float() for n in lens]
    outs = {}
    for name, kw in (("simt", {}), ("whole", PREFILL), ("cut", dict(PREFILL, scratch=1 << 20))):
        run = JointRun(spec, rel_t, talk, "cuda", torch.bfloat16, lens, form="simt" if name == "simt" else "prefill", **kw)
        first = run.step([(0, zs[0][:250], 0), (1, zs[1][:31], 0)])
        outs[name] = torch.cat([first, run.step([(1, zs[1][31:], 31), (0, zs[0][250:], 250)])])
    assert torch.equal(outs["whole"], outs["cut"])
    assert worst_row(outs["whole"].flatten(1), outs["simt"].flatten(1).cpu()) < 1e-2


# --------------------------------------------------------------------------- experts
@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("E,top,ff,H,T", [(5, 2, 40, 96, 33), (12, 3, 80, 192, 7), (1, 1, 3, 42, 2), (8, 8, 64, 64, 130), (40, 4, 100, 70, 1)])
def test_experts_are_weighed_by_their_scores_as_they_are(device, dtype, E, top, ff, H, T):
    g = torch.Generator().manual_seed(E)
    spec = MoESpec(E, top, FeedForwardSpec(ff, "silu", True), expert_weights_norm=False)
    r = lambda *s: (torch.randn(*s, generator=g) / s[-1] ** 0.5).to(dtype)
    triples = [(r(ff, H), r(ff, H), r(H, ff)) for _ in range(E)]
    router, x = r(E, H) * 0.7, torch.randn(T, H, generator=g).to(dtype)
    c, n = lambda t: t.to(device), lambda t: t.double().numpy()
    lw = LayerWeights(attn_norm=None, wqkv=None, wo=None, ffn_norm=None, experts=listed_experts(spec, [tuple(c(m) for m in t) for t in triples], H),
                      router=QTensor("F32" if dtype == torch.float32 else "BF16", c(router), tuple(router.shape)))
    w = {"router": n(router)}
    for e, t in enumerate(triples):
        w.update({f"e{e}.{name}": n(m) for name, m in zip(("gate", "up", "down"), t)})
    want = plain.experts(n(x), w, "", {"router": {"top": top}})
    if top < E:
        s = plain.choose(n(x)[0] @ n(router).T, top)[1]
        assert s.sum() < 0.95  # (dividing by the sum would show)
    assert rel(ops.moe_ffn(c(x), lw, spec), want) < (1e-2 if dtype == torch.bfloat16 else 3e-6)
    res, wn = torch.randn(T, H, generator=g), torch.rand(H, generator=g) + 0.5
    joined, _ = ops.add_normed(c(res), ops.moe_ffn(c(x), lw, spec, combine=False), c(wn), 2, 1e-5)
    assert rel(joined, n(res) + plain.grouped_norm(want, n(wn), 2, 1e-5)) < (1e-2 if dtype == torch.bfloat16 else 3e-6)


# --------------------------------------------------------------------------- pages of kept first tokens
@pytest.mark.parametrize("kept,first", [(0, 0), (1, 1), (16, 1), (17, 2), (40, 3)])
def test_pages_of_kept_first_tokens_stay(kept, first):
    """Pages behind the window go back to the pool while a sequence runs, those of kept first tokens do not; at its end all
    are free once."""
    pool = BlockPool(40, 16, enable_prefix_cache=False)
    sched = Scheduler(SchedulerConfig(64, 64, 2, attention_window=48, kept_first=kept, enable_prefix_cache=False), pool)
    seq = Sequence([], SamplingParams(temperature=0.0))
    owned = None
    for n in (40, 1, 60, 64, 1, 1, 33, 64):
        seq.prompt.extend(range(n))
        out = sched.schedule_portions([(seq, n, [])])
        before = list(seq.blocks)
        assert owned is None or before[:first] == owned
        sched.finish_portions(out)
        owned = list(before[:first])
        live = range(max(first, (seq.num_computed - 48) // 16), len(seq.blocks))
        assert [seq.blocks[i] for i in live] == [before[i] for i in live] and seq.blocks[:first] == owned
        assert pool.num_used == len(set(seq.blocks[:first]) | {seq.blocks[i] for i in live})
    assert pool.num_used < len(seq.blocks)
    sched.abort(seq.request_id)
    assert pool.num_free == 40


# --------------------------------------------------------------------------- configuration and accounting
def small():
    return plain.config(32, 20, [(plain.rwkv(2, 8, 3), plain.moe(3, 2, 8)), (plain.attn(4, 2, 8, 20, 3), plain.dense(24)), (plain.rwkv(1, 40), None),
                                 (plain.attn(2, 2, 16, 50, 18), None)], groups=4)


def test_configuration_is_read_whole(tmp_path):
    from oxidize_b200.formats.layered import LayeredCheckpoint

    cfg = small()
    path = plain.write_model(str(tmp_path / "m"), cfg, plain.random_weights(cfg))
    llm = LLM.from_checkpoint(path, EngineConfig(max_model_len=32, max_num_seqs=2), device="cpu")
    c = llm.cfg
    assert c.arch == "netovik" and c.tie_embeddings and c.embedding_scale == 3.0 and c.has_state and c.norm_groups == 4 and c.depth_average
    assert c.state_shapes == [(2, 32, 32), (1, 64, 64)] and c.state_windows == [(1, 32), (1, 32)]
    assert c.uniform_window == 50 and c.kept_first == 18 and llm.scheduler.config.kept_first == 18 and c.cache_shapes == [(2, 1, 40), (2, 1, 40)]
    a, k, m = c.layer_specs[1].mixer, c.layer_specs[0].mixer, c.layer_specs[0].ffn
    assert (a.window, a.keep_first, a.softcap, a.bias_rows, a.bias_max, a.scale) == (20, 3, 20.0, 8, 40, 0.3)
    assert a.talk and a.unit_sink and a.shared_kv and a.bias and a.qk_norm == "unit" and a.rotary is None
    assert (k.heads, k.dim, k.rank, k.hidden) == (2, 8, 3, 32) and not m.expert_weights_norm and m.expert.gated
    stored = sum(int(np.prod(t.shape)) for t in LayeredCheckpoint(path).tensors.values())
    assert c.param_count() == stored
    assert StateStore.slot_bytes(c.state_shapes, c.state_windows) * 2 == llm.kv.states.nbytes()


@pytest.mark.parametrize("change,error", [
    (lambda c: c["layers"][0].update(type="mamba"), UnsupportedArchitecture),
    (lambda c: c["layers"][0]["mlp"].update(kind="other"), UnsupportedArchitecture),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=4), ValueError),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), UnsupportedArchitecture),
    (lambda c: c["layers"][1]["mixer"].update(vdim=4), UnsupportedArchitecture),
    (lambda c: c["layers"][1]["mixer"].update(bias_max=4), UnsupportedArchitecture),
    (lambda c: c["norm"].update(groups=5), UnsupportedArchitecture)])
def test_configurations_that_are_refused(tmp_path, change, error):
    cfg = small()
    path = plain.write_model(str(tmp_path / "m"), cfg, plain.random_weights(cfg))
    change(cfg)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    with pytest.raises(error):
        LLM.from_checkpoint(path, EngineConfig(max_model_len=32), device="cpu")


def test_refusals_of_the_engine(tmp_path):
    from oxidize_b200.formats.layered import LayeredCheckpoint
    from oxidize_b200.models.layered import config_from_layered, load_layered_weights

    cfg = small()
    path = plain.write_model(str(tmp_path / "m"), cfg, plain.random_weights(cfg))
    ck = LayeredCheckpoint(path)
    with pytest.raises(ValueError):
        load_layered_weights(ck, config_from_layered(ck), tp_size=2)
    with pytest.raises(ValueError):
        LLM.from_checkpoint(path, EngineConfig(max_model_len=32, kv_cache_dtype="q8"), device="cpu")
    llm = LLM.from_checkpoint(path, EngineConfig(max_model_len=32, enable_prefix_cache=True), device="cpu")
    assert not llm.scheduler.config.enable_prefix_cache
