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
