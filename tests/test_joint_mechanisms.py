"""The mechanisms of layers whose branches read one norm, one at a time: the joint norm, query temperature, mixed values, output
gates, the gated delta rule (steps, chunks, portions, rings of convolution inputs, state slots), routed squared-relu experts with
a correction of the choice, configuration checks."""
import dataclasses
import json
import os

import numpy as np
import pytest
import torch

import pavatar_plain as plain
from oxidize_b200 import ops
from oxidize_b200.engine.kv_pool import KVCache, KVCacheSpec, StateStore
from oxidize_b200.engine.llm import LLM, EngineConfig
from oxidize_b200.models.config import AttentionSpec, DeltaSpec, FeedForwardSpec, LayerSpec, MoESpec, ParallelSpec, RotarySpec, UnsupportedArchitecture
from oxidize_b200.models.layered import delta_weights, listed_experts, pad_heads
from oxidize_b200.models.weights import LayerWeights, QTensor
from oxidize_b200.ops import ref as opref
from test_listed_mixers import B16, CPU, F32, batch, gpu, pad_rows, rel, rope_state, worst_row

TOL = {torch.float32: 2e-5, torch.bfloat16: 1.5e-2}


@pytest.fixture(autouse=True)
def _status():
    yield
    if torch.cuda.is_available():
        from oxidize_b200.ops import cuda as C

        assert C.status()[0] == 0


# --------------------------------------------------------------------------- norm
@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("T,H", [(1, 4), (5, 96), (3, 257), (7, 4096), (2, 6144), (600, 2048), (2, 10002)])
def test_both_branches_join_the_stream(device, dtype, T, H):
    g = torch.Generator().manual_seed(H + T)
    res, y0, y1, f = torch.randn(T, H, generator=g) * 3, *((torch.randn(T, H, generator=g) * s).to(dtype) for s in (0.02, 5.0, 0.7))
    w0, w1, wn = (torch.rand(H, generator=g) + 0.5 for _ in range(3))
    k = 3
    rows = torch.randn(T * k, H + 4, generator=g).to(dtype)  # routed rows may be wider than the model
    index, weights = torch.randperm(T * k, generator=g).reshape(T, k).int(), torch.rand(T, k, generator=g)
    c = lambda t: t.to(device)
    n = lambda t: t.double().numpy()
    pair = ops.NormedPair(c(y0), c(y1), c(w0), c(w1), 0.5, 0.25)
    mixes = [(None, 0.0), (c(y1), n(y1)),
             (pair, 0.5 * plain.rms_norm(n(y0), n(w0), 1e-3) + 0.25 * plain.rms_norm(n(y1), n(w1), 1e-3))]
    ffns = [(None, 0.0), (c(f), n(f))]
    if device != "cpu":
        ffns.append((ops.RoutedRows(c(rows), c(index), c(weights)), (n(rows)[index.numpy(), :H] * n(weights)[:, :, None]).sum(1)))
    for mix, wm in mixes:
        for ffn, wf in ffns:
            for nxt in (True, False):
                x, a = ops.joint_norm(c(res), mix, ffn, c(wn) if nxt else None, 1e-3, dtype)
                want = n(res) + wm + wf
                assert x.dtype == torch.float32 and rel(x, want) < 1e-6
                if nxt:
                    assert a.dtype == dtype and rel(a, plain.rms_norm(want, n(wn), 1e-3)) < (3e-3 if dtype == torch.bfloat16 else 1e-6)
                else:
                    assert a is None


# --------------------------------------------------------------------------- attention
def unrotated(H, G, d, vd, **kw):
    return AttentionSpec(H, G, d, vd, 0.3, None, bias=True, gate="head", **kw)


def attend(device, dtype, z, spec, lens, page=16, first=None, lam=None, first_width=0):
    """z [T, q | k | v | gate] unpadded rows of every sequence in one batch, each from its start; outputs [T, heads, v_dim]."""
    H, G, d, vd, W = spec.heads, spec.kv_heads, spec.dim, spec.v_dim, spec.width
    nq = H * d + G * d + G * vd
    meta, pages = batch([(n, n) for n in lens], page, device)
    kv = KVCache(KVCacheSpec(1, G, W, page, "bf16" if dtype == torch.bfloat16 else "f32"), pages, device)
    kv.data[0].fill_(3.0)
    zp = pad_rows(z[:, :nq], spec).to(device, dtype)
    gate = z[:, nq:]
    gate = (torch.nn.functional.pad(gate, (0, spec.gate_dim - H)) if spec.gate == "head" else pad_heads(gate, H, W, 1)).to(device, dtype)
    rope = None if spec.rotary is None else rope_state(spec, device)
    vf = None if first is None else pad_heads(first, G, first_width, 1).to(device, dtype).unflatten(1, (G, first_width))
    mix = None if lam is None else torch.tensor([lam], device=device)
    if device == "cpu":
        q = opref.head_prep(zp, None, None, spec, rope, meta, kv, 0, 1e-5, vf, mix)
        o = opref.head_gate(opref.paged_attention(q, kv, 0, meta, spec.scale, spec.window), gate, spec)
        return o[..., :vd]
    from oxidize_b200.ops import cuda_listed as CL

    q = CL.head_prep(zp, None, None, spec, rope, meta, kv, 0, 1e-5, vf, mix)
    o = torch.empty(z.shape[0], H * W, dtype=dtype, device=device)
    CL.attention(q, kv, 0, meta, spec, None, o, 1.0, gate)
    return o.reshape(-1, H, W)[..., :vd]


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("coef,every", [(0.7, 5), (0.5, 1), (1.3, 2.5), (0.25, 64), (0.0, 3)])
def test_query_temperature_changes_at_its_steps(device, dtype, coef, every):
    """Scores that make the factor visible, around every multiple of its period."""
    H, G, d, vd, T = 3, 1, 8, 6, 70
    spec = unrotated(H, G, d, vd, temp_coef=coef, temp_every=every)
    g = torch.Generator().manual_seed(3)
    z = torch.randn(T, (H + G) * d + G * vd + H, generator=g).to(dtype).float()
    n = z.double().numpy()
    q, k, v = n[:, : H * d].reshape(T, H, d), n[:, H * d : (H + G) * d].reshape(T, G, d), n[:, (H + G) * d : -H].reshape(T, G, vd)
    f = plain.temperature(np.arange(T), coef, every)
    assert coef == 0 or len(set(f.tolist())) == len(set(int((p + 1) // every) for p in range(T)))
    want = plain.causal(q * f[:, None, None], k, v, spec.scale) * plain.sigmoid(n[:, -H:])[:, :, None]
    assert worst_row(attend(device, dtype, z, spec, [T]), want) < TOL[dtype]


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
def test_values_are_mixed_with_the_first_layers_and_cached_mixed(device, dtype):
    """The first layer's values stand at another width than this layer's; a share of 0 and 1 keeps one of the two."""
    H, G, d, vd = 4, 2, 40, 20
    spec = unrotated(H, G, d, vd, v_mix=True)
    lens = [33, 1, 18]
    T = sum(lens)
    g = torch.Generator().manual_seed(4)
    z = torch.randn(T, (H + G) * d + G * vd + H, generator=g).to(dtype).float()
    first = torch.randn(T, G * vd, generator=g).to(dtype).float()
    for lam in (0.0, 0.35, 1.0):
        got = attend(device, dtype, z, spec, lens, first=first, lam=lam, first_width=32)
        o = 0
        for m in lens:
            n, fv = z[o : o + m].double().numpy(), first[o : o + m].double().numpy()
            q, k = n[:, : H * d].reshape(m, H, d), n[:, H * d : (H + G) * d].reshape(m, G, d)
            v = plain.mix_values(n[:, (H + G) * d : -H].reshape(m, G, vd), fv.reshape(m, G, vd), lam)
            want = plain.causal(q, k, v, spec.scale) * plain.sigmoid(n[:, -H:])[:, :, None]
            assert worst_row(got[o : o + m], want) < TOL[dtype]
            o += m


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("H,G,d,vd,rot", [(4, 2, 24, 20, 8), (3, 3, 64, 33, 64), (8, 1, 128, 128, 32), (2, 1, 10, 130, 6)])
def test_a_gate_per_output_value(device, dtype, H, G, d, vd, rot):
    spec = AttentionSpec(H, G, d, vd, 0.2, RotarySpec(rot, 1e3), gate="value")
    lens = [5, 90]
    g = torch.Generator().manual_seed(5)
    z = torch.randn(sum(lens), (H + G) * d + G * vd + H * vd, generator=g).to(dtype).float()
    got = attend(device, dtype, z, spec, lens)
    o = 0
    for m in lens:
        n = z[o : o + m].double().numpy()
        q, k = n[:, : H * d].reshape(m, H, d), n[:, H * d : (H + G) * d].reshape(m, G, d)
        v, gate = n[:, (H + G) * d : (H + G) * d + G * vd].reshape(m, G, vd), n[:, -H * vd :].reshape(m, H, vd)
        r = plain.rotation(rot, 1e3)
        want = plain.causal(plain.rotate_heads(q, r), plain.rotate_heads(k, r), v, spec.scale) * plain.sigmoid(gate)
        assert worst_row(got[o : o + m], want) < TOL[dtype]
        o += m


# --------------------------------------------------------------------------- gated delta rule
def delta_case(H, G, d, vd, taps, rd=0, rg=0, seed=0, decay=-1.5):
    """(spec, tensors as a checkpoint stores them without the projections of the input)."""
    spec = DeltaSpec(H, G, d, vd, taps, rd, rg)
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    t = {"q.conv": r(G * d, taps) / taps ** 0.5, "k.conv": r(G * d, taps) / taps ** 0.5, "v.conv": r(H * vd, taps) / taps ** 0.5,
         "A_log": r(H) - 1.0, "norm": 1 + 0.2 * r(vd), "dt_bias": r(H * d if rd else H) + decay}
    if rd:
        t["a2"] = r(H * d, rd) / rd ** 0.5
    if rg:
        t["g2"] = r(H * vd, rg) / rg ** 0.5
    for n, rows in (("q", G * d), ("k", G * d), ("v", H * vd), ("a1" if rd else "a", rd or H), ("g1" if rg else "g", rg or H * vd), ("b", H)):
        t[n] = torch.zeros(rows, 1)
    return spec, {n: x.bfloat16().float() for n, x in t.items()}


PARTS = ("q", "k", "v", "gate", "decay", "beta")


def draw(spec, T, g, dtype):
    """Projections of a sequence, unpadded, in ``dtype``'s values."""
    H, G = spec.heads, spec.kv_heads
    sizes = (G * spec.dim, G * spec.dim, H * spec.v_dim, spec.gate_rank or H * spec.v_dim, spec.decay_rank or H, H)
    return {n: torch.randn(T, s, generator=g).to(dtype).float() for n, s in zip(PARTS, sizes)}


def padded(spec, z):
    """Projections as the operators take them."""
    K, V, H, G = spec.k_width, spec.v_width, spec.heads, spec.kv_heads
    fill = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[1]))
    gate = fill(z["gate"], spec.gate_dim) if spec.gate_rank else pad_heads(z["gate"], H, V, 1)
    out = torch.cat([pad_heads(z["q"], G, K, 1), pad_heads(z["k"], G, K, 1), pad_heads(z["v"], H, V, 1), gate,
                     fill(z["decay"], spec.decay_dim), fill(z["beta"], (H + 7) // 8 * 8)], 1)
    assert out.shape[1] == spec.proj_dim
    return out


def delta_plain(spec, t, z, eps=1e-5):
    """(outputs [T, heads, v_dim], final states [heads, dim, v_dim]) of a whole sequence."""
    H, G, d, vd = spec.heads, spec.kv_heads, spec.dim, spec.v_dim
    n = {k: v.double().numpy() for k, v in z.items()}
    w = {k: v.double().numpy() for k, v in t.items()}
    T = len(n["q"])
    q, k, v = (plain.silu(plain.short_conv(n[c], w[c + ".conv"])) for c in "qkv")
    q, k, v = plain.unit(q.reshape(T, G, d)) * d ** -0.5, plain.unit(k.reshape(T, G, d)), v.reshape(T, H, vd)
    a = n["decay"] @ w["a2"].T if spec.decay_rank else n["decay"]
    g = np.exp(-np.exp(w["A_log"])[None, :, None] * plain.softplus(a + w["dt_bias"]).reshape(T, H, -1))
    beta = plain.sigmoid(n["beta"])
    gate = plain.sigmoid(n["gate"] @ w["g2"].T) if spec.gate_rank else plain.silu(n["gate"])
    heads = [plain.delta_scan(q[:, h // (H // G)], k[:, h // (H // G)], v[:, h], g[:, h], beta[:, h]) for h in range(H)]
    o = np.stack([x for x, _ in heads], 1)
    return plain.unit_rms(o, eps) * w["norm"] * gate.reshape(T, H, vd), np.stack([s for _, s in heads])


class DeltaRun:
    """Sequences fed portion by portion through the operator, each with its own slot."""

    def __init__(self, spec, t, device, dtype, slots=6, **kw):
        self.spec, self.device, self.dtype, self.kw = spec, device, dtype, kw
        _, w = delta_weights(spec, t, dtype)
        move = lambda x: None if x is None else x.to(device)
        self.w = dataclasses.replace(w, **{f.name: move(getattr(w, f.name)) for f in dataclasses.fields(w)})
        self.store = StateStore([spec.state_shape], slots, device, [spec.window_shape])
        self.store.data[0].fill_(7.0)  # nothing of an earlier owner may be seen
        self.store.windows[0].fill_(-5.0)

    def step(self, parts):
        """``parts``: (projections of the rows fed, rows before them, slot); outputs of all rows, unpadded."""
        spec = self.spec
        z = torch.cat([padded(spec, z) for z, _, _ in parts]).to(self.device, self.dtype)
        lens = [(len(z["q"]), past + len(z["q"])) for z, past, _ in parts]
        meta, _ = batch(lens, 16, self.device, slots=[s for _, _, s in parts])
        if self.device == "cpu":
            out = opref.delta_rule(z, self.w, spec, meta, self.store.data[0], self.store.windows[0], 1e-5)
        else:
            from oxidize_b200.ops import cuda_delta

            out = torch.full((z.shape[0], spec.out_dim), float("nan"), dtype=self.dtype, device=self.device)
            cuda_delta.delta_rule(z, self.w, spec, meta, self.store.data[0], self.store.windows[0], 1e-5, out, **self.kw)
        out = out.reshape(-1, spec.heads, spec.v_width)
        assert not out[..., spec.v_dim :].any()
        return out[..., : spec.v_dim]

    def feed(self, z, cuts, slot=2):
        out, at = [], 0
        for n in cuts:
            out.append(self.step([({k: v[at : at + n] for k, v in z.items()}, at, slot)]))
            at += n
        assert at == len(z["q"])
        return torch.cat(out)

    def state(self, slot=2):
        return self.store.data[0][slot][:, : self.spec.dim, : self.spec.v_dim]


STATE_TOL = {torch.float32: 1e-5, torch.bfloat16: 4e-5}
SHAPES = [  # heads, q / k heads, dim, vdim, taps, ranks of decay and gate
    (4, 2, 24, 20, 4, 0, 0), (4, 4, 64, 48, 3, 40, 24), (1, 1, 1, 1, 1, 0, 0), (3, 1, 128, 128, 4, 33, 16), (2, 2, 96, 112, 2, 0, 40),
    (2, 1, 33, 48, 5, 7, 0), (2, 2, 160, 64, 4, 8, 8), (6, 3, 32, 128, 7, 0, 0), (2, 2, 128, 16, 4, 0, 0), (1, 1, 64, 200, 3, 16, 16)]


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("shape", SHAPES, ids=str)
def test_delta_rule_however_a_sequence_is_cut(device, dtype, shape):
    """Whole, token by token, in portions that end anywhere in a chunk and in a convolution: outputs and the final state."""
    spec, t = delta_case(*shape)
    T = 150
    z = draw(spec, T, torch.Generator().manual_seed(1), dtype)
    want, state = delta_plain(spec, t, z)
    for cuts in ([T], [1] * T, [2, 3] * 30, [1, 64, 1, 63, 21], [100, 1, 1, 48], [9, 8] * 8 + [14]):
        run = DeltaRun(spec, t, device, dtype)
        got = run.feed(z, cuts)
        assert worst_row(got, want) < TOL[dtype], cuts
        assert rel(run.state(), state) < STATE_TOL[dtype], cuts
        assert (run.store.data[0][3] == 7.0).all() and (run.store.windows[0][3] == -5.0).all()


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("rank", [0, 8])
def test_delta_rule_with_decays_of_every_strength(device, dtype, rank):
    """Tokens that forget (nearly) everything, tokens that forget nothing, and runs of both, at any place of a chunk: no
    exponent may overflow, and what lies behind a forgetting token stays exact."""
    spec, t = delta_case(2, 1, 32, 32, 3, rank, 0)
    t["A_log"] = torch.tensor([2.0, -3.0])
    T = 200
    g = torch.Generator().manual_seed(2)
    z = draw(spec, T, g, dtype)
    z["decay"] *= 4.0
    z["decay"][torch.randperm(T, generator=g)[:20]] *= 10.0
    z["decay"][70:90] = -60.0 if not rank else z["decay"][70:90]
    z["decay"][[3, 47, 48, 63, 64, 130]] *= 30.0
    z["decay"] = z["decay"].to(dtype).float()
    want, state = delta_plain(spec, t, z)
    for cuts in ([T], [1] * T, [65, 65, 70]):
        run = DeltaRun(spec, t, device, dtype)
        got = run.feed(z, cuts)
        assert torch.isfinite(got.float()).all() and worst_row(got, want) < 2 * TOL[dtype]
        assert rel(run.state(), state) < STATE_TOL[dtype]


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
def test_delta_rule_remembers_far_writes(device, dtype):
    """No decay but for what the key itself overwrites: one value written under a key of its own is read 300 tokens later."""
    spec, t = delta_case(1, 1, 64, 32, 1, 0, 0)
    t["A_log"], t["dt_bias"] = torch.tensor([-20.0]), torch.tensor([-9.0])
    for c in "qkv":
        t[c + ".conv"] = torch.ones_like(t[c + ".conv"])
    T = 330
    z = draw(spec, T, torch.Generator().manual_seed(3), dtype)
    key = torch.zeros(64)
    key[5] = 8.0
    z["k"][:, 5] = -30.0  # (silu: nothing along this channel)
    z["k"][17], z["q"][320] = key, key
    z["k"][17, 6:] = z["q"][320, 6:] = -30.0
    z["v"][17] = 9.0
    want, _ = delta_plain(spec, t, z)
    hidden = {k: v.clone() for k, v in z.items()}
    hidden["v"][17] = -9.0
    assert worst_row(want[320], delta_plain(spec, t, hidden)[0][320]) > 0.5  # (the read-out hangs on that write)
    for cuts in ([T], [18, 1, 200, 101, 10], [300] + [1] * 30):
        got = DeltaRun(spec, t, device, dtype).feed(z, cuts)
        assert worst_row(got[320], want[320]) < TOL[dtype] and worst_row(got, want) < 2 * TOL[dtype]


@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
def test_delta_rule_batches_and_reused_slots(device, dtype):
    """Long and short portions and single tokens of several sequences in one step, a padding row without a slot, and slots
    that a new sequence takes over."""
    spec, t = delta_case(4, 2, 64, 48, 4, 16, 16)
    g = torch.Generator().manual_seed(6)
    zs = [draw(spec, n, g, dtype) for n in (170, 12, 40, 75)]
    wants = [delta_plain(spec, t, z)[0] for z in zs]
    run = DeltaRun(spec, t, device, dtype)
    part = lambda i, lo, hi: ({k: v[lo:hi] for k, v in zs[i].items()}, lo)
    plan = [[(0, 0, 70), (1, 0, 1), (2, 0, 33)], [(2, 33, 34), (0, 70, 71), (1, 1, 8)], [(1, 8, 9), (2, 34, 35), (0, 71, 72)],
            [(0, 72, 170), (2, 35, 40), (1, 9, 12)], [(3, 0, 75)]]
    slots = {0: 4, 1: 0, 2: 5, 3: 4}
    got = {i: [] for i in slots}
    for entries in plan:
        out = run.step([part(*e) + (slots[e[0]],) for e in entries] + [part(1, 0, 1) + (-1,)])
        o = 0
        for i, lo, hi in entries:
            got[i].append(out[o : o + hi - lo])
            o += hi - lo
        assert not out[o:].any()
    for i in slots:
        assert worst_row(torch.cat(got[i]), wants[i]) < TOL[dtype], i


@gpu
@pytest.mark.parametrize("values,rounds", [(16, 1), (32, 2), (32, 100)])
@pytest.mark.parametrize("shape", [s for s in SHAPES if s[3] <= 128 and s[2] <= 128], ids=str)
def test_chunks_agree_with_steps(shape, values, rounds):
    """The tensor-core kernels, in rounds of any number of chunks, against the token-by-token one on the same 16-bit rows, and
    twice the same."""
    spec, t = delta_case(*shape, seed=3)
    if spec.v_width % values:
        pytest.skip("not a multiple")
    z = draw(spec, 333, torch.Generator().manual_seed(9), torch.bfloat16)
    for cuts in ([333], [64, 128, 141], [9, 55, 269]):
        runs = [DeltaRun(spec, t, "cuda", torch.bfloat16, chunk_rows=r, values=values, rounds=rounds) for r in (2, 2, 1 << 20)]
        outs = [r.feed(z, cuts) for r in runs]
        assert torch.equal(outs[0], outs[1]) and torch.equal(runs[0].state(), runs[1].state())
        assert rel(runs[0].state(), runs[2].state()) < 4e-5 and worst_row(outs[0], outs[2].cpu()) < 1e-2
        assert torch.equal(runs[0].store.windows[0], runs[2].store.windows[0])


# --------------------------------------------------------------------------- experts
@pytest.mark.parametrize("device,dtype", [CPU, F32, B16])
@pytest.mark.parametrize("E,top,ff,H,T", [(5, 2, 40, 96, 33), (12, 3, 80, 192, 7), (1, 1, 3, 42, 2), (8, 8, 64, 64, 130), (40, 4, 100, 70, 1)])
def test_squared_relu_experts_with_a_correction(device, dtype, E, top, ff, H, T):
    """The correction changes who is chosen and not what the chosen weigh."""
    g = torch.Generator().manual_seed(E)
    spec = MoESpec(E, top, FeedForwardSpec(ff, "relu2"), expert_weights_scale=1.7, correction=True)
    r = lambda *s: (torch.randn(*s, generator=g) / s[-1] ** 0.5).to(dtype)
    ups, downs, router, x = [r(ff, H) for _ in range(E)], [r(H, ff) for _ in range(E)], r(E, H) * 3, torch.randn(T, H, generator=g).to(dtype)
    corr = torch.randn(E, generator=g) * 0.3
    c = lambda t: t.to(device)
    ex = listed_experts(spec, [(None, c(u), c(d)) for u, d in zip(ups, downs)], H)
    lw = LayerWeights(attn_norm=None, wqkv=None, wo=None, ffn_norm=None, experts=ex, router_bias=c(corr),
                      router=QTensor("F32" if dtype == torch.float32 else "BF16", c(router), tuple(router.shape)))
    n = lambda t: t.double().numpy()
    w = {"router": n(router), "correction": n(corr)}
    for e in range(E):
        w[f"e{e}.up"], w[f"e{e}.down"] = n(ups[e]), n(downs[e])
    want = plain.experts(n(x), w, "", {"router": {"top": top, "scale": 1.7}})
    if 1 < top < E and T > 1:
        z = n(x) @ n(router).T
        assert any(set(plain.choose(row, n(corr), top, 1)[0]) != set(plain.choose(row, 0.0, top, 1)[0]) for row in z)
    got = ops.moe_ffn(c(x), lw, spec)
    assert rel(got, want) < (1e-2 if dtype == torch.bfloat16 else 3e-6)
    res, wn = torch.randn(T, H, generator=g), torch.rand(H, generator=g) + 0.5
    joined, _ = ops.joint_norm(c(res), None, ops.moe_ffn(c(x), lw, spec, combine=False), c(wn), 1e-5, dtype)
    assert rel(joined, n(res) + want) < (1e-2 if dtype == torch.bfloat16 else 3e-6)


# --------------------------------------------------------------------------- configuration and accounting
def small():
    return plain.config(32, 20, [(plain.dlt(2, 1, 8, 8, 3), plain.moe(3, 2, 8)), (plain.attn(2, 1, 8, 8, (0.5, 4)), None),
                                 (plain.parallel(plain.rotated(2, 1, 8, 8, plain.rotation(8)), plain.dlt(2, 2, 4, 4, 2)), None),
                                 (plain.attn(2, 1, 16, 8), None)])


def test_configuration_is_read_whole(tmp_path):
    cfg = small()
    path = plain.write_model(str(tmp_path / "m"), cfg, plain.random_weights(cfg, rank=5))
    llm = LLM.from_checkpoint(path, EngineConfig(max_model_len=32, max_num_seqs=2), device="cpu")
    c = llm.cfg
    assert c.arch == "pavatar" and c.tie_embeddings and c.embedding_scale == 3.0 and c.final_softcap == 20.0 and c.has_state
    assert c.state_shapes == [(2, 32, 16), (2, 32, 16)] and c.state_windows == [(3, 96), (2, 160)] and c.uniform_window == 0
    a, p = c.layer_specs[1].mixer, c.layer_specs[2].mixer
    assert (a.temp_coef, a.temp_every, a.v_mix, a.gate, a.bias, a.rotary) == (0.5, 4.0, True, "head", True, None)
    assert isinstance(p, ParallelSpec) and p.norms and p.left.qk_norm == "head" and p.left.gate == "value" and (p.right.decay_rank, p.right.gate_rank) == (5, 5)
    stored = sum(int(np.prod(t.shape)) for t in __import__("oxidize_b200.formats.layered", fromlist=["x"]).LayeredCheckpoint(path).tensors.values())
    assert c.param_count() == stored
    assert StateStore.slot_bytes(c.state_shapes, c.state_windows) * 2 == llm.kv.states.nbytes()


@pytest.mark.parametrize("change,error", [
    (lambda c: c["layers"][0].update(type="mamba"), UnsupportedArchitecture),
    (lambda c: c["layers"][0]["mlp"].update(kind="other"), UnsupportedArchitecture),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=4), ValueError),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), UnsupportedArchitecture),
    (lambda c: c["layers"][0]["mixer"].update(conv=0), ValueError),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), UnsupportedArchitecture),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=0), ValueError),
    (lambda c: c["layers"][3]["mixer"].update(vdim=4), ValueError),
    (lambda c: c["layers"][2]["mixer"]["left"]["rot"].update(dims=7), UnsupportedArchitecture),
    (lambda c: c["layers"][2]["mixer"]["left"]["rot"].update(dims=10), UnsupportedArchitecture)])
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
    llm = LLM.from_checkpoint(path, EngineConfig(max_model_len=32, enable_prefix_cache=True), device="cpu")
    assert not llm.scheduler.config.enable_prefix_cache
    assert LayerSpec(DeltaSpec(2, 1, 8, 8, 3)).attention is None
