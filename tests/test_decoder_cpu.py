"""The plain decoder implementation (oracle/decoder.py) shows the faults that the GPU tests look for: each
mechanism left out or shifted by one changes the output by far more than the tests tolerate. And what of the
product runs on the host: the distance buckets, the config reader, the trace replay."""
import ctypes as C
import json
import math

import numpy as np
import pytest

from oracle import decoder as D
import decoder_util as U
import vkllama_b200 as vk
from vkllama_b200.trace import replay


def outputs(cfg, W, toks, **over):
    return D.run(cfg, W, toks, **over)


def attention_with(**over):
    return lambda h, W, p, mix: D.attention_mixer(h, W, p, mix, **over)


MIX = U.config([(U.attn(6, 2, 24, bias_max=40, every=9), U.dense(100, 0.9)), (U.attn(4, 1, 40, bias_max=60), U.moe(32, 5, 2))], width=88,
               loop={"start": 0, "stop": 2, "times": 2})


def shifted_bias(table, far, n):
    return np.stack([table[D.distance_bucket(k + 1, table.shape[0], far)] for k in range(n + 1)])


def wrong_edge(table, far, n):  # the first half of the buckets ends one distance late
    half = table.shape[0] // 2
    return np.stack([table[D.distance_bucket(k - (k == half), table.shape[0], far)] for k in range(n + 1)])


@pytest.mark.parametrize("fault", [
    attention_with(temp_of=lambda p, c, e: np.ones(len(p))),
    attention_with(temp_of=lambda p, c, e: D.query_temperature(p - 1, c, e)),
    attention_with(bias_of=lambda t, far, n: np.zeros((n + 1, t.shape[1]))),
    attention_with(bias_of=shifted_bias),
    attention_with(bias_of=wrong_edge),
    attention_with(bias_of=lambda t, far, n: D.distance_bias(t, far + 8, n)),
])
def test_attention_faults_show(fault):
    W, toks = U.weights(MIX, 1), U.tokens(MIX, 90, 2)
    want = outputs(MIX, W, toks)
    assert U.rel_err(outputs(MIX, W, toks, mixer=fault), want) > 20 * U.REL["float32"]


@pytest.mark.parametrize("drop", ["l0.mix.g", "l0.mix.q.b", "l0.mix.k.b", "l1.mix.o.b", "l0.norm1.b", "final.norm.b", "loop.step"])
def test_missing_weights_show(drop):
    W, toks = U.weights(MIX, 1), U.tokens(MIX, 60, 2)
    want = outputs(MIX, W, toks)
    V = dict(W)
    V[drop] = np.zeros_like(W[drop])
    assert U.rel_err(outputs(MIX, V, toks), want) > 2 * U.REL["bfloat16"]


def test_feed_forward_faults_show():
    W, toks = U.weights(MIX, 1), U.tokens(MIX, 60, 2)
    want = outputs(MIX, W, toks)

    def ff(mod):
        def f(h, W, p, mlp, tokens):
            m = dict(mlp)
            if mod == "limit" and mlp["kind"] == "dense":
                m["limit"] = 1e9
            if mod == "table" and mlp["kind"] == "moe":
                tokens = (np.asarray(tokens) + 1) % MIX["vocab"]
            return D.feed_forward(h, W, p, m, tokens)
        return f

    for mod in ("limit", "table"):
        assert U.rel_err(outputs(MIX, W, toks, ff=ff(mod)), want) > 2 * U.REL["bfloat16"], mod


def test_loop_order_shows():
    W, toks = U.weights(MIX, 1), U.tokens(MIX, 40, 2)
    want = outputs(MIX, W, toks)
    assert D.layer_runs(MIX) == [(0, 0), (1, 0), (0, 1), (1, 1)]
    V = dict(W)
    V["loop.step"] = W["loop.step"][::-1]
    assert U.rel_err(outputs(MIX, V, toks), want) > 2 * U.REL["bfloat16"]


@pytest.mark.parametrize("rows,far", [(32, 200), (32, 256), (20, 50), (24, 96), (16, 512), (6, 27), (2, 5), (64, 4096), (9, 30)])
def test_distance_buckets(rows, far):
    got = [vk.distance_bucket(n, rows, far) for n in range(far + 40)]
    assert got == [D.distance_bucket(n, rows, far) for n in range(far + 40)]
    h = rows // 2
    assert got[:h] == list(range(h)) and got[far:] == [rows - 1] * 40 and all(b - a in (0, 1) or a < rows - 1 for a, b in zip(got, got[1:]))
    for n in range(h, far):  # the defining formula, away from exact powers
        v = math.log(n / h) / math.log(far / h) * (rows - h)
        if abs(v - round(v)) > 1e-6:
            assert got[n] == min(rows - 1, h + math.floor(v))


def test_distance_bucket_starts_are_exact():
    # 16 * 2^k with far = 16 * 2^4: distances that are exactly the first of their bucket
    assert [vk.distance_bucket(n, 32, 256) for n in (31, 32, 63, 64, 127, 128, 255, 256)] == [19, 20, 23, 24, 27, 28, 31, 31]
    assert vk.distance_bucket(3, 8, 4) == -1  # a table that is longer than its reach


def test_the_standout_key_matters_at_every_distance():
    cfg, W = U.standout()
    for dist in U.DISTANCES:
        for at in (0, 64):
            toks = U.standout_tokens(cfg, at, dist)
            want = D.run(cfg, W, toks)[-1:]
            hidden = toks.copy()
            hidden[at] = 5
            assert U.rel_err(D.run(cfg, W, hidden)[-1:], want) > 2.5 * U.REL["bfloat16"], (dist, at)
    # and so does the row of the table that its distance names, where the row changes
    for dist in (1, 7, 8, 130 - 1):
        toks = U.standout_tokens(cfg, 0, dist)
        want = D.run(cfg, W, toks)[-1:]
        V = dict(W)
        V["l0.mix.rel"] = W["l0.mix.rel"].copy()
        V["l0.mix.rel"][D.distance_bucket(dist, 16, 130)] -= 3.0
        assert U.rel_err(D.run(cfg, V, toks)[-1:], want) > 20 * U.REL["float32"], dist


def create(text):
    L = vk.load_library()
    out = C.c_void_p()
    st = L.vkl_model_create_config(None, text.encode(), 64, vk.FP32, C.byref(out))
    return st, L.vkl_last_error().decode()


def test_config_reader():
    assert vk.architectures() == ["Rumalorn", "Kupuzen"]
    for cfg in U.CASES.values():
        st, msg = create(json.dumps(cfg))
        assert st == 3 and "null device" in msg  # the config itself was taken
    good = json.dumps(MIX)
    assert create(good[:-1])[1].startswith("config: malformed JSON")
    assert create(good.replace("Rumalorn", "Unknown"))[0] == 12
    assert create("{}")[0] == 3

    def broken(change):
        c = json.loads(good)
        change(c)
        return create(json.dumps(c))

    assert "vocab" in broken(lambda c: c.pop("vocab"))[1]
    assert "layers" in broken(lambda c: c.pop("layers"))[1]
    assert broken(lambda c: c["layers"][0].update(type="other"))[0] == 12
    assert "vdim" in broken(lambda c: c["layers"][0]["mixer"].update(vdim=7))[1] or "width" in broken(lambda c: c["layers"][0]["mixer"].update(vdim=7))[1]
    assert "bias_max" in broken(lambda c: c["layers"][0]["mixer"].pop("bias_max"))[1]
    assert "limit" in broken(lambda c: c["layers"][0]["mlp"].pop("limit"))[1]
    assert broken(lambda c: c["layers"][1]["mlp"].update(kind="other"))[0] == 12
    assert "whole" in broken(lambda c: c.update(width=3.5))[1]
    ok = broken(lambda c: c.update(loop=None, note="é\n"))
    assert "null device" in ok[1]


class FakeModel:
    def __init__(self):
        self.calls = []

    def forward_rows(self, toks, pos, rows):
        self.calls.append((list(toks), pos, list(rows)))
        return np.array([[toks[r], pos + r] for r in rows], np.float32).reshape(len(rows), 2)


def test_trace_replay(tmp_path):
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 6, 7], "want": [0, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [8], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": [9], "want": [0]}], "end": ["b"]}]
    m, said = FakeModel(), []
    replay(m, [json.dumps(s) for s in steps] + ["\n"], str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"]
    assert m.calls == [([5, 6, 7], 0, [0, 2]), ([8], 3, []), ([9], 0, [0])]
    assert np.fromfile(tmp_path / "0.f32", "<f4").tolist() == [5, 0, 7, 2]
    assert not (tmp_path / "1.f32").exists()
    assert np.fromfile(tmp_path / "2.f32", "<f4").tolist() == [9, 0]
    with pytest.raises(ValueError):
        replay(m, [json.dumps(steps[0]), json.dumps(steps[2])], str(tmp_path), said.append)


def test_checkpoint_writer_round_trip(tmp_path):
    W = U.weights(MIX, 4)
    back = D.write_folder(str(tmp_path), MIX, W)
    read = D.read_safetensors(str(tmp_path / "model.safetensors"))
    assert set(read) == set(W)
    for k in W:
        assert np.array_equal(read[k], back[k]) and np.array_equal(back[k], W[k]), k
