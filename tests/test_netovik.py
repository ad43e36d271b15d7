"""Netovik through the engine against the plain statement in ``netovik_plain``: whole prompts, portions, decoding, batches,
reused pages and state slots, generation.  The same cases run on the CPU path and, on a GPU box, on the device in float32 and
bfloat16."""
import functools
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import netovik_plain as plain
from oxidize_b200.engine.llm import LLM, EngineConfig
from oxidize_b200.engine.replay import TraceReplay
from oxidize_b200.engine.sampler import SamplingParams
from test_sokirax import PATHS, check, engine, feed, gpu, spread

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CONFIGS = {
    # layers of different geometry, windows and tables; kept first tokens that end inside a page, at its end and past it
    "varied": plain.config(96, 203, [
        (plain.rwkv(4, 24), plain.moe(5, 2, 40)),
        (plain.attn(6, 2, 24, 30, 5, 15.0, 12, 50), plain.dense(72)),
        (plain.rwkv(3, 40, 17), None),
        (plain.attn(5, 5, 16, 48, 16, 8.0, 32, 64, 0.5), plain.moe(9, 3, 24)),
        (plain.attn(8, 4, 32, 17, 21, 30.0, 4, 300, 0.2), plain.moe(4, 1, 88)),
        (plain.rwkv(2, 60, 3), plain.dense(33))], groups=3),
    # sizes and constants of one, and sizes that are no multiple of anything
    "ones": plain.config(42, 51, [
        (plain.attn(1, 1, 2, 1, 1, 5.0, 2, 2, 1.0), plain.moe(1, 1, 1)),
        (plain.rwkv(1, 1, 1), plain.moe(2, 1, 3)),
        (plain.attn(3, 1, 7, 2, 0, 1.0, 2, 90), plain.dense(1)),
        (plain.rwkv(5, 7, 2), plain.moe(3, 2, 10)),
        (plain.attn(7, 7, 33, 40, 3), None)], groups=1, eps=1e-3, embed_scale=1.0),
    # wide heads, whole parts of 128 values, a window beyond every prompt
    "wide": plain.config(256, 90, [
        (plain.rwkv(2, 128, 32), plain.dense(192)),
        (plain.attn(8, 2, 96, 64, 4, 25.0, 32, 128, 0.12), plain.moe(8, 2, 64)),
        (plain.rwkv(4, 64, 16), plain.moe(8, 2, 64)),
        (plain.attn(4, 4, 128, 1000, 0, 50.0, 16, 90, 0.1), plain.moe(8, 2, 64))], embed_scale=11.3),
}


@functools.lru_cache(None)
def weights(name):
    return plain.random_weights(CONFIGS[name], seed=sum(map(ord, name)))


@functools.lru_cache(None)
def oracle(name, tokens):
    return plain.forward(CONFIGS[name], weights(name), list(tokens))


def prompt(name, n, seed=1):
    return tuple(np.random.default_rng(seed).integers(0, CONFIGS[name]["vocab"], n).tolist())


@pytest.fixture(scope="module")
def model_dirs(tmp_path_factory):
    base = tmp_path_factory.mktemp("netovik")
    return {n: plain.write_model(str(base / n), CONFIGS[n], weights(n)) for n in CONFIGS}


@pytest.fixture(autouse=True)
def _status():
    yield
    if torch.cuda.is_available():
        from oxidize_b200.ops import cuda as C

        assert C.status()[0] == 0


@pytest.mark.parametrize("device,dtype", PATHS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt(model_dirs, name, device, dtype):
    toks = prompt(name, 150)
    rep = TraceReplay(engine(model_dirs[name], device, dtype, 192))
    check(feed(rep, toks, [150]), oracle(name, toks)[1], dtype)
    if dtype == "float32":
        check(feed(rep, toks[:1], [1]), oracle(name, toks)[1][:1], dtype, "one token")


@pytest.mark.parametrize("device,dtype", PATHS)
@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("cuts", [[1], [2], [2, 3], [17, 1, 30], [16], [64, 2], [9, 8], [129, 3, 1]])
def test_portions_and_token_by_token(model_dirs, name, cuts, device, dtype):
    """However a prompt is cut, every position's logits are those of the whole sequence."""
    n = 150 if device != "cpu" else 90
    toks = prompt(name, 150)[:n]
    rep = TraceReplay(engine(model_dirs[name], device, dtype, 192))
    check(feed(rep, toks, spread(n, cuts)), oracle(name, prompt(name, 150))[1][:n], dtype)


@pytest.mark.parametrize("device,dtype", PATHS)
def test_pages_of_other_sizes(model_dirs, device, dtype):
    toks = prompt("varied", 150)
    for page in (8, 32, 64, 4):
        rep = TraceReplay(engine(model_dirs["varied"], device, dtype, 192, page))
        check(feed(rep, toks, [40, 1, 1, 2, 106]), oracle("varied", toks)[1], dtype, f"page {page}")


@pytest.mark.parametrize("device,dtype", PATHS)
@pytest.mark.parametrize("name", ["varied", "wide"])
def test_unequal_requests_in_one_batch(model_dirs, name, device, dtype):
    """Portions of some requests beside single tokens of others, requests that pause, and a pool in which pages and state
    slots are used again; each request against its own oracle."""
    lens = {"a": 90, "b": 33, "c": 1, "d": 164, "e": 45, "f": 70, "g": 2}
    seqs = {k: prompt(name, n, seed=ord(k)) for k, n in lens.items()}
    rep = TraceReplay(engine(model_dirs[name], device, dtype, 448))
    rng = np.random.default_rng(5)
    waiting, live, at, got = list(lens), [], {k: 0 for k in lens}, {k: [] for k in lens}
    for _ in range(400):
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
        if not live:
            break
        entries, end = [], []
        for k in live:
            if rng.random() < 0.25:
                continue
            n = min(int(rng.choice([1, 1, 2, 3, 16, 29, 80])), lens[k] - at[k])
            entries.append({"id": k, "tokens": seqs[k][at[k] : at[k] + n], "want": list(range(n))})
            at[k] += n
            if at[k] == lens[k]:
                end.append(k)
        rng.shuffle(entries)
        logits = rep.step(entries, end)
        o = 0
        for e in entries:
            got[e["id"]].append(logits[o : o + len(e["tokens"])])
            o += len(e["tokens"])
        live = [k for k in live if k not in end]
    assert not live and not waiting and rep.llm.pool.num_free == rep.llm.pool.num_blocks
    assert len(rep.llm.scheduler.slots.free) == 4
    if dtype == "bfloat16":  # (all rows together: a request of one token has no rows to let off)
        check(torch.cat([torch.cat(got[k]) for k in lens]), np.concatenate([oracle(name, seqs[k])[1] for k in lens]), dtype)
        return
    for k in lens:
        check(torch.cat(got[k]), oracle(name, seqs[k])[1], dtype, k)


@pytest.mark.parametrize("device,dtype", PATHS)
def test_freed_pages_and_slots_do_not_leak_into_the_next_request(model_dirs, device, dtype):
    """A pool of one request's size: every request lands on the pages, and in the state slot, of the one before."""
    rep = TraceReplay(engine(model_dirs["wide"], device, dtype, 128))
    for seed, cuts in ((3, [50, 2, 1, 47]), (4, [1] * 30 + [70]), (5, [100])):
        toks = prompt("wide", 100, seed)
        check(feed(rep, toks, cuts), oracle("wide", toks)[1], dtype, str(seed))
        assert rep.llm.pool.num_free == rep.llm.pool.num_blocks and len(rep.llm.scheduler.slots.free) == 4
    with pytest.raises(RuntimeError):
        rep.step([{"id": "x", "tokens": prompt("wide", 128), "want": []}, {"id": "y", "tokens": [1], "want": []}], [])


@pytest.mark.parametrize("device,dtype", PATHS)
def test_long_decoding_with_pages_handed_back(model_dirs, device, dtype):
    """Every layer is windowed: pages behind the widest window go back to the pool while the request runs, those of the kept
    first tokens stay, and another request takes the ones that were given back."""
    n = 260
    toks, other = prompt("varied", n, 9), prompt("varied", 100, 10)
    llm = engine(model_dirs["varied"], device, dtype, 320)
    assert llm.scheduler.config.attention_window == 48 and llm.scheduler.config.kept_first == 21
    rep = TraceReplay(llm)
    got = [feed(rep, toks[:200], [20] + [1] * 180, end=False)]
    assert llm.pool.num_used <= 2 + 48 // 16 + 2
    out = []
    for t in range(60):
        entries = [{"id": "a", "tokens": [toks[200 + t]], "want": [0]}]
        if t < 50:
            entries.append({"id": "b", "tokens": other[2 * t : 2 * t + 2], "want": [0, 1]})
        lg = rep.step(entries, (["b"] if t == 49 else []) + (["a"] if t == 59 else []))
        got.append(lg[:1])
        out.append(lg[1:])
    check(torch.cat(got), oracle("varied", toks)[1], dtype)
    check(torch.cat(out), oracle("varied", other)[1], dtype)
    assert llm.pool.num_free == llm.pool.num_blocks


@pytest.mark.parametrize("device,dtype", PATHS)
def test_what_every_layer_hands_on(model_dirs, device, dtype):
    from oxidize_b200.models.transformer import BatchMeta

    toks = prompt("varied", 150)[:60]
    llm = engine(model_dirs["varied"], device, dtype, 64)
    i32 = dict(dtype=torch.int32, device=llm.device)
    pos = torch.arange(60, **i32)
    meta = BatchMeta(torch.tensor(toks, **i32), pos, pos.clone(), torch.tensor([0, 60], **i32), torch.tensor([60], **i32),
                     torch.arange(4, **i32)[None, :], pos.clone(), 60, 60, 1, state_slots=torch.tensor([2], **i32))
    layers = range(len(CONFIGS["varied"]["layers"]))
    cap = {"layers": set(layers)}
    h, _ = llm.model.run_layers(llm.model.embed(meta.token_ids), None, meta, llm.kv, capture=cap)
    assert h.dtype == torch.float32
    want = oracle("varied", prompt("varied", 150))[0][:, :60]
    for i in layers:
        assert cap["hidden"][i].dtype == torch.float32
        check(cap["hidden"][i], want[i], dtype, f"layer {i}")


# --------------------------------------------------------------------------- generation
@pytest.mark.parametrize("device,dtype", PATHS[:2])
def test_greedy_generation_through_the_scheduler(model_dirs, device, dtype):
    """LLM.generate: chunked prefill, continuous batching, decoding (captured on the GPU); every generated token is the
    oracle's, or one whose logit is within rounding of it."""
    llm = LLM.from_checkpoint(model_dirs["varied"], EngineConfig(max_model_len=128, max_num_seqs=3, num_kv_blocks=24,
                              max_num_batched_tokens=32, prefill_chunk_size=11, compute_dtype="f32"), device=device)
    prompts = [list(prompt("varied", n, 20 + n)) for n in (5, 40, 17, 29, 1)]
    for _ in range(2):  # the second time on used pages and slots (and captured graphs)
        outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True))
        for p, o in zip(prompts, outs):
            assert len(o.token_ids) == 24
            lg = oracle("varied", tuple(p + o.token_ids))[1]
            for j, t in enumerate(o.token_ids):
                row = lg[len(p) - 1 + j]
                assert row[t] > row.max() - 1e-3 * row.std(), (len(p), j)
    assert len(llm.scheduler.slots.free) == 3


@pytest.mark.parametrize("device,dtype", [pytest.param("cuda:0", "bfloat16", marks=gpu)])
def test_generation_in_16_bits_with_and_without_captured_graphs(model_dirs, device, dtype):
    prompts = [list(prompt("wide", n, 50 + n)) for n in (9, 65, 30)]
    sp = SamplingParams(temperature=0.0, max_tokens=40, ignore_eos=True)
    base = dict(max_model_len=160, max_num_seqs=4, num_kv_blocks=48, max_num_batched_tokens=64, prefill_chunk_size=32)
    got = []
    for graphs in (True, False):
        llm = LLM.from_checkpoint(model_dirs["wide"], EngineConfig(cuda_graphs=graphs, **base), device=device)
        got.append([o.token_ids for o in llm.generate(prompts, sp)])
        assert bool(llm.runner.graphs) == graphs
    near = total = 0
    for p, toks in zip(prompts, got[0]):  # near the oracle's choice
        lg = oracle("wide", tuple(p + toks))[1]
        for j, t in enumerate(toks):
            row = lg[len(p) - 1 + j]
            near, total = near + (row[t] > row.max() - 0.25 * row.std()), total + 1
    assert near >= 0.9 * total
    same = sum(a == b for x, y in zip(*got) for a, b in zip(x, y))
    assert same >= 0.7 * 120  # (key splits differ between the two, and with them the rounding)


@pytest.mark.parametrize("device,dtype", PATHS[:2])
def test_preempted_requests_generate_the_same(model_dirs, device, dtype):
    """A pool too small for all requests: a preempted one gives its slot back and starts again from nothing; prefixes are
    never shared, since a state cannot be rebuilt from pages."""
    sp = SamplingParams(temperature=0.0, max_tokens=20, ignore_eos=True)
    head = list(prompt("varied", 40, 77))
    prompts = [head + [3], head + [4, 5], list(prompt("varied", 30, 78))]

    def run(**kw):
        llm = LLM.from_checkpoint(model_dirs["varied"], EngineConfig(max_model_len=128, max_num_seqs=3, max_num_batched_tokens=64,
                                  prefill_chunk_size=16, compute_dtype="f32", **kw), device=device)
        return [o.token_ids for o in llm.generate(prompts, sp)], llm

    want, _ = run(num_kv_blocks=64)
    again, tight = run(num_kv_blocks=9)
    assert again == want and tight.scheduler.num_preemptions > 0 and len(tight.scheduler.slots.free) == 3
    assert not tight.scheduler.config.enable_prefix_cache and tight.pool.hits == 0


def test_streamed_layers_and_sampling(model_dirs):
    """Layers loaded as the forward pass reaches them, and seeded sampling."""
    sp = SamplingParams(temperature=0.8, top_k=20, seed=7, max_tokens=12, ignore_eos=True)
    got = []
    for resident in (0, 2):
        llm = LLM.from_checkpoint(model_dirs["varied"], EngineConfig(max_model_len=64, max_num_seqs=2, resident_layers=resident),
                                  device="cpu")
        got.append([o.token_ids for o in llm.generate([list(prompt("varied", 10, 3)), [5]], sp)])
    assert got[0] == got[1]


def test_command_line_generates(model_dirs):
    toks = prompt("varied", 9, 4)
    cmd = [sys.executable, "-m", "oxidize_b200.cli.main", "run", model_dirs["varied"], "--tokens", ",".join(map(str, toks)),
           "--backend", "cpu", "--temperature", "0", "--max-tokens", "6", "--no-auto", "--ctx-size", "64"]
    r = subprocess.run(cmd, capture_output=True, text=True, cwd=ROOT, timeout=300)
    assert r.returncode == 0, r.stderr
    got = [int(t) for t in r.stdout.split()]
    assert got == plain.greedy(CONFIGS["varied"], weights("varied"), toks, 6)
    show = subprocess.run(cmd[:3] + ["show", model_dirs["varied"]], capture_output=True, text=True, cwd=ROOT, timeout=300)
    assert show.returncode == 0 and json.loads(show.stdout)["architecture"] == "netovik"


def test_random_weights_of_its_shapes_run():
    """Drawn weights pass through the same layouts as loaded ones."""
    from oxidize_b200.models.registry import config_from_checkpoint
    from oxidize_b200.utils.synth import synth_weights
    from oxidize_b200.formats.layered import LayeredCheckpoint

    import tempfile

    with tempfile.TemporaryDirectory() as d:
        cfg = config_from_checkpoint(LayeredCheckpoint(plain.write_model(d, CONFIGS["varied"], weights("varied"))))
    llm = LLM(synth_weights(cfg, torch.device("cpu"), "F32", seed=1), EngineConfig(max_model_len=64, max_num_seqs=2, num_kv_blocks=8, compute_dtype="f32"))
    outs = llm.generate([[1, 2, 3]], SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True))
    assert len(outs[0].token_ids) == 5


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_program(model_dirs, tmp_path, dtype):
    """bin/trace_run: steps on standard input, one answer line each, logits of the wanted places on disk."""
    a, b = prompt("wide", 100, 31), prompt("wide", 25, 32)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:77], "want": [0, 76]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:20], "want": [5]}, {"id": "a", "tokens": a[77:78], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[78:80], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[80:], "want": [19]}, {"id": "b", "tokens": b[20:], "want": [4, 0]}],
              "end": ["a", "b"]}]
    want = {0: [("a", 0), ("a", 76)], 1: [("b", 5), ("a", 77)], 3: [("a", 99), ("b", 24), ("b", 20)]}
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", model_dirs["wide"], "--dtype", dtype, "--out",
                        str(tmp_path), "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps),
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    assert sorted(os.listdir(tmp_path)) == ["0.f32", "1.f32", "3.f32"]
    lg = {"a": oracle("wide", a)[1], "b": oracle("wide", b)[1]}
    got = [torch.from_numpy(np.fromfile(tmp_path / f"{s}.f32", dtype="<f4").reshape(len(rows), -1)) for s, rows in want.items()]
    check(torch.cat(got), np.stack([lg[i][p] for rows in want.values() for i, p in rows]), dtype)
