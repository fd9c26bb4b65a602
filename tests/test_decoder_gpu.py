"""Layer-list decoder designs on the GPU against the plain implementation in oracle/decoder.py, through the
framework's own model driver: whole prompts, portions, token by token, sequence after sequence in the same
caches, keys that stand out at chosen distances, greedy and sampled generation, and the folder loader."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import decoder as D
import decoder_util as U
import vkllama_b200 as vk
from vkllama_b200.__main__ import generate
from vkllama_b200.trace import replay

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
COMPUTE = {"float32": vk.FP32, "bfloat16": vk.BF16}


def load(dev, cfg, W, maxlen, dtype):
    m = vk.Model.from_config(dev, cfg, maxlen, COMPUTE[dtype])
    for k, v in W.items():
        if v.dtype.kind in "iu":
            m.set_weight(k, vk.UINT32, v.astype(np.int32))
        else:
            m.set_weight(k, vk.BF16, D.f32_to_bf16(v.reshape(-1)))
    return m


def run_portions(m, toks, sizes, start=0):
    """Logits of every token, fed in portions (the last size repeats)."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(k, len(sizes) - 1)], len(toks) - at)
        out.append(m.forward_rows(toks[at:at + n], start + at, np.arange(n)))
        at, k = at + n, k + 1
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(U.CASES))
def test_every_layer_and_logit(dev, name, dtype):
    """Each branch of the design with sizes of its own: the residual stream after every layer run and all logits."""
    cfg = U.CASES[name]
    W, toks = U.weights(cfg, 11), U.tokens(cfg, 150, 12)
    layers = []
    want = D.run(cfg, W, toks, layers_out=layers)
    m = load(dev, cfg, W, 160, dtype)
    got = m.trace_layers(toks)
    assert got.shape[0] == len(layers) == len(D.layer_runs(cfg))
    for r, (a, b) in enumerate(zip(got, layers)):
        assert U.rel_err(a, b) < U.REL[dtype], "layer run %d" % r
    assert U.rel_err(m.forward_rows(toks, 0, np.arange(len(toks))), want) < U.REL[dtype]
    # a token of its own: the one-token kernels leave the same stream
    one = m.trace_layers(toks[-1:], len(toks) - 1)
    assert U.rel_err(one[:, 0], np.stack(layers)[:, -1]) < U.REL[dtype]
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["loop inside", "loop from the first layer", "wide heads"])
def test_portions_and_single_tokens_agree_with_the_whole_prompt(dev, name, dtype):
    cfg = U.CASES[name]
    W, toks = U.weights(cfg, 21), U.tokens(cfg, 200, 22)
    want = D.run(cfg, W, toks)
    m = load(dev, cfg, W, 200, dtype)
    for sizes in ([200], [1], [2], [3, 64, 2, 15, 17, 16, 1], [63, 65], [128, 2], [199, 1]):
        assert U.rel_err(run_portions(m, toks, sizes), want) < U.REL[dtype], sizes
    m.close()


def test_32bit_results_do_not_depend_on_the_cut(dev):
    cfg = U.CASES["loop inside"]
    W, toks = U.weights(cfg, 23), U.tokens(cfg, 140, 24)
    m = load(dev, cfg, W, 140, "float32")
    whole = run_portions(m, toks, [140])
    for sizes in ([1], [2], [5, 70, 2]):
        assert U.rel_err(run_portions(m, toks, sizes), whole) < U.REL["float32"]
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sequences_one_after_another_in_the_same_caches(dev, dtype):
    """Unequal sequences, long before short and short before long: none sees what another left."""
    cfg = U.CASES["loop from the first layer"]
    W = U.weights(cfg, 31)
    m = load(dev, cfg, W, 260, dtype)
    for i, (n, sizes) in enumerate([(250, [250]), (1, [1]), (33, [2]), (180, [90, 1]), (2, [1]), (64, [64]), (20, [20])]):
        toks = U.tokens(cfg, n, 40 + i)
        assert U.rel_err(run_portions(m, toks, sizes), D.run(cfg, W, toks)) < U.REL[dtype], n
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_key_that_stands_out_at_every_kind_of_distance(dev, dtype):
    """The matching key sits just inside and outside the one-by-one buckets, the saturation distance, the 64-row
    tiles and at the sequence's first tokens; the query in a prompt, in a portion and decoded alone."""
    cfg, W = U.standout()
    m = load(dev, cfg, W, 400, dtype)
    for dist in U.DISTANCES:
        for at in (0, 1, 63, 64):
            toks = U.standout_tokens(cfg, at, dist)
            n = len(toks)
            want = D.run(cfg, W, toks)[-1:]
            assert U.rel_err(m.forward_rows(toks, 0, [n - 1]), want) < U.REL[dtype], (dist, at)
            assert U.rel_err(m(toks[-1:], n - 1)[None], want) < U.REL[dtype], (dist, at, "decoded")
            if n > 40:
                m.forward_rows(toks[:n - 20], 0, [])
                assert U.rel_err(m.forward_rows(toks[n - 20:], n - 20, [19]), want) < U.REL[dtype], (dist, at, "portion")
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dev, dtype):
    cfg = U.CASES["one pass"]
    W, toks = U.weights(cfg, 61), U.tokens(cfg, 700, 62)
    want = D.run(cfg, W, toks)
    m = load(dev, cfg, W, 700, dtype)
    m.forward_rows(toks[:3], 0, [])
    got = np.stack([m(toks[i:i + 1], i) for i in range(3, 700)])
    assert U.rel_err(got, want[3:]) < U.REL[dtype]
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_many_tokens_per_expert_and_experts_without_tokens(dev, dtype):
    cfg = U.config([(U.attn(4, 2, 16), U.moe(48, 6, 2))], width=64, vocab=50)
    W = U.weights(cfg, 71)
    W["l0.mlp.table"][:30] = [4, 1]      # most tokens share two experts, over several 128-row tiles
    W["l0.mlp.table"][30:] = [0, 4]      # experts 2, 3 and 5 have none
    m = load(dev, cfg, W, 600, dtype)
    for n in (2, 129, 300, 600):
        toks = U.tokens(cfg, n, n)
        assert U.rel_err(m.forward_rows(toks, 0, np.arange(n)), D.run(cfg, W, toks)) < U.REL[dtype], n
    m.close()


def greedy(cfg, W, prompt, n):
    """The oracle's greedy ids and the smallest gap between its first and second choice, over the logits' spread."""
    toks, gap = list(prompt), np.inf
    for _ in range(n):
        y = D.run(cfg, W, toks)[-1]
        top = np.sort(y)[-2:]
        gap = min(gap, (top[1] - top[0]) / y.std())
        toks.append(int(np.argmax(y)))
    return toks[len(prompt):], gap


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["loop inside", "loop from the first layer"])
def test_greedy_generation(dev, name, dtype):
    """vkl_model_generate (prompt pass, then replays of the captured decode step) and the per-token loop."""
    cfg, n, W = U.CASES[name], 16, U.weights(U.CASES[name], 81)
    need = {"float32": 1e-3, "bfloat16": 0.03}[dtype]
    for seed in range(40):  # a prompt whose every step is decided by more than the type's rounding
        prompt = U.tokens(cfg, 30, seed)
        ids, gap = greedy(cfg, W, prompt, n)
        if gap > need:
            break
    else:
        pytest.fail("no decided prompt")
    m = load(dev, cfg, W, 64, dtype)
    assert m.generate(prompt, n)[0].tolist() == ids
    assert m.generate(prompt[:1], 3)[0].tolist() == [int(t) for t in m.generate(prompt[:1], 3)[0]]
    assert m.generate(prompt, n)[0].tolist() == ids  # the graph of the first call, the caches in use
    tok, got = prompt, []
    for i in range(n):
        y = m(tok, 0 if i == 0 else len(prompt) + i - 1)
        got.append(int(np.argmax(y)))
        assert m.last_token() == got[-1]
        vals, top = m.topk(4)
        assert top[0] == got[-1] and np.array_equal(vals, np.sort(y)[::-1][:4])
        tok = np.array(got[-1:], np.uint32)
    assert got == ids
    assert generate(m, prompt, n) == ids == generate(m, prompt, n, topk=1, seed=3)
    sampled = generate(m, prompt, n, topk=8, seed=5)
    assert sampled == generate(m, prompt, n, topk=8, seed=5) and len(set(sampled)) > 1
    assert generate(m, prompt, 4, topp=0.5, seed=5) == generate(m, prompt, 4, topp=0.5, seed=5)
    m.close()


def test_folder_command_line_and_trace(dev, tmp_path):
    cfg = U.CASES["loop from the first layer"]
    W, toks = U.weights(cfg, 91), U.tokens(cfg, 40, 92)
    folder = str(tmp_path / "model")
    D.write_folder(folder, cfg, W)
    want = D.run(cfg, W, toks)
    m = vk.load_model(dev, folder, 64, vk.FP32)
    assert U.rel_err(m.forward_rows(toks, 0, np.arange(40)), want) < U.REL["float32"]
    said = []
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:25].tolist(), "want": [0, 24]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[25:26].tolist(), "want": [0]}], "end": ["x"]}]
    replay(m, [json.dumps(s) for s in steps], str(tmp_path), said.append)
    y = np.fromfile(tmp_path / "0.f32", "<f4").reshape(2, -1)
    assert U.rel_err(y, want[[0, 24]]) < U.REL["float32"]
    assert U.rel_err(np.fromfile(tmp_path / "1.f32", "<f4")[None], want[25:26]) < U.REL["float32"]
    ids = m.generate(toks[:8], 6)[0].tolist()
    m.close()
    out = subprocess.run([sys.executable, "-m", "vkllama_b200", "generate", "--model", folder, "--maxlen", "64", "--dtype", "float32", "--tokens", "6",
                          "--prompt", ",".join(str(t) for t in toks[:8])], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr
    assert [int(t) for t in out.stdout.split()] == ids
    run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "bfloat16", "--out", str(tmp_path), "--max-tokens", "64"],
                         input=json.dumps(steps[0]) + "\n", capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr
    assert "done 0" in run.stdout.splitlines()
    assert U.rel_err(np.fromfile(tmp_path / "0.f32", "<f4").reshape(2, -1), want[[0, 24]]) < U.REL["bfloat16"]


def test_refusals(dev, tmp_path):
    cfg = U.CASES["experts"]
    W = U.weights(cfg, 95)
    m = vk.Model.from_config(dev, cfg, 32, vk.BF16)
    with pytest.raises(vk.VklError) as e:
        m(np.array([1], np.uint32), 0)
    assert e.value.code == 9 and "is not set" in e.value.message
    with pytest.raises(vk.VklError):
        m.set_weight("l0.mix.v", vk.BF16, np.zeros(4, np.uint16))
    with pytest.raises(vk.VklError):
        m.set_weight("embed", vk.BF16, np.zeros(4, np.uint16))
    with pytest.raises(vk.VklError):
        m.set_weight("l0.mlp.table", vk.UINT32, np.full_like(W["l0.mlp.table"], 3))  # three experts: 0, 1, 2
    m.close()
    m = load(dev, cfg, W, 32, "bfloat16")
    for bad in (lambda: m.forward_rows(U.tokens(cfg, 33), 0, []), lambda: m(np.array([1], np.uint32), 32),
                lambda: m.generate(U.tokens(cfg, 30), 3), lambda: m(np.array([cfg["vocab"]], np.uint32), 0),
                lambda: m.forward_rows(U.tokens(cfg, 4), 0, [4])):
        with pytest.raises(vk.VklError) as e:
            bad()
        assert e.value.code == 11
    m.close()
    W["l0.mix.q"] = W["l0.mix.q"].T.copy()  # same bytes, another shape
    D.write_folder(str(tmp_path), cfg, W)
    with pytest.raises(vk.VklError) as e:
        vk.load_model(dev, str(tmp_path), 32)
    assert "l0.mix.q" in e.value.message


def test_synthetic_weights_run_and_use_a_cache_of_keys_only(dev):
    cfg = U.CASES["dense"]
    m = vk.Model.from_config(dev, cfg, 48, vk.BF16)
    m.synth_weights(7)
    y = m.forward_rows(U.tokens(cfg, 20), 0, np.arange(20))
    assert np.isfinite(y).all() and y.std() > 0
    assert m.kv_shape(0) == (4, 48, 16) and m.cache_bytes() == 4 * 48 * 16 * 2
    k, _ = m.read_kv(0)
    assert (k[:, :20] != 0).any() and not k[:, 20:].any()
    m.close()
