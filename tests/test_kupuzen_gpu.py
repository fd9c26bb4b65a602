"""Kupuzen on the GPU against the plain implementation in oracle/decoder.py, through the framework's own model driver:
every branch with sizes of its own, whole prompts, portions, token by token, sequence after sequence in the same caches
and states, keys just inside and outside a window, writes that a state has to keep, greedy and sampled generation,
and the folder loader. The driver holds one sequence at a time, so unequal sequences follow one another."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import decoder as D
import kupuzen_util as U
import vkllama_b200 as vk
from vkllama_b200.__main__ import generate

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
COMPUTE = {"float32": vk.FP32, "bfloat16": vk.BF16}
DTYPES = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])


def load(dev, case, W, maxlen, dtype):
    m = vk.Model.from_config(dev, case[0], maxlen, COMPUTE[dtype], shapes=U.shapes(W))
    for k, v in W.items():
        m.set_weight(k, vk.BF16, D.f32_to_bf16(v.reshape(-1)))
    return m


def run_portions(m, toks, sizes):
    """Logits of every token, fed in portions (the last size repeats)."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(k, len(sizes) - 1)], len(toks) - at)
        out.append(m.forward_rows(toks[at:at + n], at, np.arange(n)))
        at, k = at + n, k + 1
    return np.concatenate(out)


@DTYPES
@pytest.mark.parametrize("name", list(U.CASES))
def test_every_layer_and_logit(dev, name, dtype):
    """The residual stream after every layer and all logits, from a whole prompt and from its tokens one by one."""
    case = U.CASES[name]
    W, toks = U.weights(case, 11), U.tokens(case[0], 150, 12)
    layers = []
    want = D.run(case[0], W, toks, layers_out=layers)
    m = load(dev, case, W, 160, dtype)
    got = m.trace_layers(toks)
    assert got.shape[0] == len(layers)
    for r, (a, b) in enumerate(zip(got, layers)):
        assert U.rel_err(a, b) < U.REL[dtype], "layer %d" % r
    assert U.rel_err(m.forward_rows(toks, 0, np.arange(len(toks))), want) < U.REL[dtype]
    m.forward_rows(toks[:100], 0, [])
    one = np.concatenate([m.trace_layers(toks[i:i + 1], i) for i in range(100, 150)], axis=1)
    for r, (a, b) in enumerate(zip(one, layers)):
        assert U.rel_err(a, b[100:]) < U.REL[dtype], "layer %d, decoded" % r
    m.close()


@DTYPES
@pytest.mark.parametrize("name", ["mixed", "attention around delta", "shared caches", "wide delta", "wide heads"])
def test_portions_and_single_tokens_agree_with_the_whole_prompt(dev, name, dtype):
    case = U.CASES[name]
    W, toks = U.weights(case, 21), U.tokens(case[0], 200, 22)
    want = D.run(case[0], W, toks)
    m = load(dev, case, W, 200, dtype)
    for sizes in ([200], [1], [2], [3], [3, 64, 2, 15, 17, 16, 1], [63, 65], [128, 2], [199, 1], [1, 199]):
        assert U.rel_err(run_portions(m, toks, sizes), want) < U.REL[dtype], sizes
    m.close()


def test_32bit_results_do_not_depend_on_the_cut(dev):
    case = U.CASES["mixed"]
    W, toks = U.weights(case, 23), U.tokens(case[0], 140, 24)
    m = load(dev, case, W, 140, "float32")
    whole = run_portions(m, toks, [140])
    for sizes in ([1], [2], [5, 70, 2]):
        assert U.rel_err(run_portions(m, toks, sizes), whole) < U.REL["float32"]
    m.close()


@DTYPES
def test_sequences_one_after_another_in_the_same_caches_and_states(dev, dtype):
    """Unequal sequences, long before short and short before long: none sees what another left."""
    case = U.CASES["attention around delta"]
    W = U.weights(case, 31)
    m = load(dev, case, W, 260, dtype)
    for i, (n, sizes) in enumerate([(250, [250]), (1, [1]), (33, [2]), (180, [90, 1]), (2, [1]), (64, [64]), (20, [20]), (7, [3, 1])]):
        toks = U.tokens(case[0], n, 40 + i)
        assert U.rel_err(run_portions(m, toks, sizes), D.run(case[0], W, toks)) < U.REL[dtype], n
    m.close()


def test_a_new_sequence_leaves_the_same_states_as_a_fresh_model(dev):
    case = U.CASES["delta, many heads per key"]
    W, toks = U.weights(case, 33), U.tokens(case[0], 50, 34)
    m, used = load(dev, case, W, 120, "float32"), load(dev, case, W, 120, "float32")
    used.forward_rows(U.tokens(case[0], 111, 35), 0, [])
    for x in (m, used):
        x.forward_rows(toks[:30], 0, [])
        for i in range(30, 50):
            x(toks[i:i + 1], i)
    assert np.array_equal(m.read_state(0), used.read_state(0)) and np.abs(m.read_state(0)).max() > 0.1
    m.close()
    used.close()


@DTYPES
def test_a_key_that_stands_out_around_the_windows_edge(dev, dtype):
    """The matching key just inside and outside the window, at the 64-row tiles' borders and at the sequence's first
    tokens; the query in a prompt, in a portion and decoded alone."""
    case, W = U.standout()
    m = load(dev, case, W, 400, dtype)
    for dist in U.DISTANCES:
        for at in (0, 1, 63, 64):
            toks = U.standout_tokens(case, at, dist)
            n = len(toks)
            want = D.run(case[0], W, toks)[-1:]
            assert U.rel_err(m.forward_rows(toks, 0, [n - 1]), want) < U.REL[dtype], (dist, at)
            assert U.rel_err(m(toks[-1:], n - 1)[None], want) < U.REL[dtype], (dist, at, "decoded")
            if n > 40:
                m.forward_rows(toks[:n - 20], 0, [])
                assert U.rel_err(m.forward_rows(toks[n - 20:], n - 20, [19]), want) < U.REL[dtype], (dist, at, "portion")
    m.close()


@DTYPES
def test_a_write_that_the_state_has_to_keep(dev, dtype):
    case, W = U.keeping()
    m = load(dev, case, W, 500, dtype)
    for dist in (1, 2, 7, 8, 9, 30, 129, 400):
        toks = U.standout_tokens(case, 3, dist)
        n = len(toks)
        want = D.run(case[0], W, toks)[-1:]
        assert U.rel_err(m.forward_rows(toks, 0, [n - 1]), want) < U.REL[dtype], dist
        m.forward_rows(toks[:n - 1], 0, [])
        assert U.rel_err(m(toks[-1:], n - 1)[None], want) < U.REL[dtype], (dist, "decoded")
        m.forward_rows(toks[:4], 0, [])
        if n > 6:
            m.forward_rows(toks[4:n - 2], 4, [])
            assert U.rel_err(m.forward_rows(toks[n - 2:], n - 2, [1]), want) < U.REL[dtype], (dist, "portions")
    m.close()


@DTYPES
def test_long_decoding(dev, dtype):
    """Windows pass over decoded tokens many times, states are carried for hundreds of steps."""
    case = U.CASES["mixed"]
    W, toks = U.weights(case, 61), U.tokens(case[0], 600, 62)
    want = D.run(case[0], W, toks)
    m = load(dev, case, W, 600, dtype)
    m.forward_rows(toks[:3], 0, [])
    got = np.stack([m(toks[i:i + 1], i) for i in range(3, 600)])
    assert U.rel_err(got, want[3:]) < U.REL[dtype]
    m.close()


@DTYPES
def test_prompts_of_more_than_a_thousand_tokens_and_many_heads(dev, dtype):
    """Longer than the delta rule's slices, and state columns enough to fill the GPU's SMs."""
    case = U.config([(U.delta(40, 20, 64, 64, 4, (6, 11)), 48), (U.delta(10, 5, 100, 256, 4, (13, 5)), None)], width=64, vocab=70)
    W, toks = U.weights(case, 63), U.tokens(case[0], 1090, 64)
    want = D.run(case[0], W, toks)
    m = load(dev, case, W, 1090, dtype)
    for sizes in ([1090], [7, 1030, 2, 50, 1], [1024, 64, 1]):
        assert U.rel_err(run_portions(m, toks, sizes), want) < U.REL[dtype], sizes
    m.close()


def test_a_stream_too_wide_for_the_norm_inside_the_decode_projection(dev):
    case = U.config([(U.attn(2, 1, 32, 32, 9, 8), 24), (U.delta(2, 1, 32, 16, 4, (5, 5)), 16)], width=6016, vocab=40)
    W, toks = U.weights(case, 67), U.tokens(case[0], 30, 68)
    want = D.run(case[0], W, toks)
    m = load(dev, case, W, 30, "float32")
    for sizes in ([30], [20, 1]):
        assert U.rel_err(run_portions(m, toks, sizes), want) < U.REL["float32"], sizes
    assert m.generate(toks[:20], 2)[0][0] == np.argmax(want[19])
    m.close()


def test_a_decode_window_that_is_split_over_several_ctas(dev):
    case = U.config([(U.attn(8, 2, 32, 32, 700, 32), 64)], width=64, vocab=60)
    W, toks = U.weights(case, 65), U.tokens(case[0], 1000, 66)
    want = D.run(case[0], W, toks)
    for dtype in ("float32", "bfloat16"):
        m = load(dev, case, W, 1000, dtype)
        m.forward_rows(toks[:990], 0, [])
        got = np.stack([m(toks[i:i + 1], i) for i in range(990, 1000)])
        assert U.rel_err(got, want[990:]) < U.REL[dtype]
        m.close()


def greedy(case, W, prompt, n):
    """The oracle's greedy ids and the smallest gap between its first and second choice, over the logits' spread."""
    toks, gap = list(prompt), np.inf
    for _ in range(n):
        y = D.run(case[0], W, toks)[-1]
        top = np.sort(y)[-2:]
        gap = min(gap, (top[1] - top[0]) / y.std())
        toks.append(int(np.argmax(y)))
    return toks[len(prompt):], gap


@DTYPES
@pytest.mark.parametrize("name", ["mixed", "delta, many heads per key"])
def test_greedy_generation(dev, name, dtype):
    """vkl_model_generate (prompt pass, then replays of the captured decode step) and the per-token loop."""
    case, n = U.CASES[name], 12
    W = U.weights(case, 81)
    need = {"float32": 1e-3, "bfloat16": 0.03}[dtype]
    for seed in range(40):  # a prompt whose every step is decided by more than the type's rounding
        prompt = U.tokens(case[0], 30, seed)
        ids, gap = greedy(case, W, prompt, n)
        if gap > need:
            break
    else:
        pytest.fail("no decided prompt")
    m = load(dev, case, W, 64, dtype)
    assert m.generate(prompt, n)[0].tolist() == ids
    assert m.generate(prompt[:1], 3)[0].tolist() == [int(t) for t in m.generate(prompt[:1], 3)[0]]
    assert m.generate(prompt, n)[0].tolist() == ids  # the graph of the first call, caches and states in use
    last = np.array(ids[-1:], np.uint32)             # the sequence goes on where generation left it
    assert U.rel_err(m(last, 30 + n - 1)[None], D.run(case[0], W, list(prompt) + ids)[-1:]) < U.REL[dtype]
    tok, got = prompt, []
    for i in range(n):
        y = m(tok, 0 if i == 0 else len(prompt) + i - 1)
        got.append(int(np.argmax(y)))
        assert m.last_token() == got[-1]
        tok = np.array(got[-1:], np.uint32)
    assert got == ids
    assert generate(m, prompt, n) == ids == generate(m, prompt, n, topk=1, seed=3)
    assert generate(m, prompt, n, topk=8, seed=5) == generate(m, prompt, n, topk=8, seed=5)
    m.close()


def test_folder_command_line_and_trace(dev, tmp_path):
    case = U.CASES["mixed"]
    W, toks = U.weights(case, 91), U.tokens(case[0], 40, 92)
    W["l2.norm2"] = np.zeros(136, np.float32)  # a layer without a feed-forward may bring its norm all the same
    folder = str(tmp_path / "model")
    D.write_folder(folder, case[0], W)
    want = D.run(case[0], W, toks)
    m = vk.load_model(dev, folder, 64, vk.FP32)
    assert U.rel_err(m.forward_rows(toks, 0, np.arange(40)), want) < U.REL["float32"]
    ids = m.generate(toks[:8], 6)[0].tolist()
    m.close()
    out = subprocess.run([sys.executable, "-m", "vkllama_b200", "generate", "--model", folder, "--maxlen", "64", "--dtype", "float32", "--tokens", "6",
                          "--prompt", ",".join(str(t) for t in toks[:8])], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr
    assert [int(t) for t in out.stdout.split()] == ids
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:25].tolist(), "want": [0, 24]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[25:27].tolist(), "want": [1]}], "end": ["x"]},
             {"step": 2, "entries": [{"id": "y", "tokens": toks[:3].tolist(), "want": [2]}], "end": ["y"]}]
    run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "bfloat16", "--out", str(tmp_path), "--max-tokens", "64"],
                         input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr
    assert [x for x in run.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    for step, rows in ((0, [0, 24]), (1, [26]), (2, [2])):
        y = np.fromfile(tmp_path / ("%d.f32" % step), "<f4").reshape(len(rows), -1)
        assert U.rel_err(y, want[rows]) < U.REL["bfloat16"], step


def test_refusals(dev):
    case = U.CASES["mixed"]
    W, toks = U.weights(case, 95), U.tokens(case[0], 20, 96)
    m = vk.Model.from_config(dev, case[0], 32, vk.BF16, shapes=U.shapes(W))
    with pytest.raises(vk.VklError) as e:
        m(toks[:1], 0)
    assert e.value.code == 9 and "is not set" in e.value.message
    for name in ("l3.mix.k", "l3.mix.v", "l3.mix.k.norm", "l0.mix.sink", "l1.mix.q.b", "l0.norm1.b"):  # not tensors of these layers
        with pytest.raises(vk.VklError):
            m.set_weight(name, vk.BF16, np.zeros(4, np.uint16))
    m.close()
    m = load(dev, case, W, 32, "bfloat16")
    m.forward_rows(toks[:10], 0, [])
    for offset in (9, 11):  # a state is at one position only
        with pytest.raises(vk.VklError) as e:
            m(toks[:1], offset)
        assert e.value.code == 9 and "10 tokens" in e.value.message
    m(toks[10:11], 10)
    m.forward_rows(toks[:2], 0, [])  # or starts anew
    m.decode_profile(1, 5)           # leaves the states at no position
    with pytest.raises(vk.VklError):
        m(toks[2:3], 2)
    m.forward_rows(toks[:2], 0, [])
    m.close()
    other = json.loads(json.dumps(case[0]))
    other["layers"][3]["mixer"]["kv_from"] = 0  # a layer without keys
    with pytest.raises(vk.VklError):
        vk.Model.from_config(dev, other, 32, vk.BF16, shapes=U.shapes(W))


def test_synthetic_weights_and_what_a_layer_keeps(dev):
    case = U.CASES["mixed"]
    W = U.weights(case, 97)
    m = vk.Model.from_config(dev, case[0], 48, vk.BF16, shapes=U.shapes(W))
    m.synth_weights(7)
    y = m.forward_rows(U.tokens(case[0], 20), 0, np.arange(20))
    assert np.isfinite(y).all() and y.std() > 0
    assert m.cache_info(1)[:4] == (3, 48, 32, 48) and m.cache_info(3)[:4] == (0, 0, 0, 0)
    assert m.cache_info(0)[5:9] == (4, 32, 64, 4) and m.read_state(0).shape == (4, 32, 64)
    k, v = m.read_kv(1)
    assert (k[:, :20, :20] != 0).any() and not k[:, 20:].any() and (v[:, :20, :36] != 0).any() and not v[:, 20:].any()
    with pytest.raises(vk.VklError):
        m.read_kv(0)
    m.close()
