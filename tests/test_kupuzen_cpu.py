"""The plain Kupuzen implementation (oracle/decoder.py) shows the faults that the GPU tests look for: each mechanism
left out, shifted by one or done in another order changes the output by far more than the tests tolerate. And what of
the product runs on the host: the config reader and the shapes it takes from the checkpoint."""
import ctypes as C
import json

import numpy as np
import pytest

from oracle import decoder as D
import kupuzen_util as U
import vkllama_b200 as vk

MIX = U.CASES["mixed"]
ATTEND = lambda **over: lambda *a, **k: D.causal_attention(*a, **{**k, **{n: f(k[n]) for n, f in over.items()}})


def attention(**over):
    return {"attention": lambda *a: D.windowed_mixer(*a, **over)}


def delta(**over):
    return {"delta": lambda *a: D.delta_mixer(*a, **over)}


def split_halves(x, pos, freq):
    n = len(freq)
    order = np.arange(2 * n).reshape(2, n).T.reshape(-1)  # pairs (i, i + n) as neighbours
    y = x.copy()
    y[..., order] = D.rotate_pairs(x[..., order], pos, freq)
    return y


def scalar_decay(q, k, v, g, beta):
    return D.delta_recurrence(q, k, v, np.repeat(g.mean(-1, keepdims=True), g.shape[-1], -1), beta)


def read_before_write(q, k, v, g, beta):
    T, H, d = q.shape
    S, out = np.zeros((H, d, v.shape[2])), np.zeros(v.shape)
    for t in range(T):
        S = g[t][:, :, None] * S
        out[t] = np.einsum("hde,hd->he", S, q[t])
        S = S + k[t][:, :, None] * (beta[t][:, None] * (v[t] - np.einsum("hde,hd->he", S, k[t])))[:, None, :]
    return out


def decay_after_write(q, k, v, g, beta):
    return D.delta_recurrence(q, k, v, np.concatenate([np.ones_like(g[:1]), g[:-1]]), beta)


def lost_state(q, k, v, g, beta):  # a portion of 40 tokens, then a fresh state
    return np.concatenate([D.delta_recurrence(*(x[:40] for x in (q, k, v, g, beta))), D.delta_recurrence(*(x[40:] for x in (q, k, v, g, beta)))])


def lost_taps(x, taps):
    return np.concatenate([D.short_convolution(x[:40], taps), D.short_convolution(x[40:], taps)])


@pytest.mark.parametrize("fault", [
    attention(attend=ATTEND(window=lambda w: w + 1)),
    attention(attend=ATTEND(window=lambda w: w - 1)),
    attention(attend=ATTEND(window=lambda w: None)),
    attention(attend=ATTEND(sink=lambda s: None)),
    attention(attend=ATTEND(sink=lambda s: s * 0.3)),
    attention(attend=ATTEND(sink=lambda s: s + np.log(2.0))),
    attention(turn=lambda x, p, f: x),
    attention(turn=lambda x, p, f: D.rotate_pairs(x, -p, f)),
    attention(turn=split_halves),
    attention(freq_of=lambda base, dims, s: D.rotation_frequencies(base, dims)),
    attention(freq_of=lambda base, dims, s: D.rotation_frequencies(base, dims, dict(s, low=s["high"] * 0.999))),
    delta(recur=scalar_decay), delta(recur=read_before_write), delta(recur=decay_after_write), delta(recur=lost_state),
    delta(conv=lost_taps), delta(conv=lambda x, t: D.short_convolution(x, t[:, ::-1])), delta(conv=lambda x, t: x * t[:, -1]),
    delta(unit_of=lambda x: x),
])
def test_mixer_faults_show(fault):
    W, toks = U.weights(MIX, 1), U.tokens(MIX[0], 90, 2)
    assert U.rel_err(D.run(MIX[0], W, toks, **fault), D.run(MIX[0], W, toks)) > 20 * U.REL["float32"]


def test_rotating_everything_after_the_keys_are_shared():
    """A layer that uses another's cache turns its own queries only: with keys of its own it would differ."""
    W, toks = U.weights(MIX, 1), U.tokens(MIX[0], 60, 2)
    want = D.run(MIX[0], W, toks)
    cfg = json.loads(json.dumps(MIX[0]))
    del cfg["layers"][3]["mixer"]["kv_from"]
    V = dict(W, **{"l3.mix." + k: W["l1.mix." + k] for k in ("k", "k.norm", "v")})
    assert U.rel_err(D.run(cfg, V, toks), want) > 2 * U.REL["bfloat16"]


@pytest.mark.parametrize("drop", ["l0.norm1", "l0.norm2", "final.norm", "l1.mix.q.norm", "l1.mix.k.norm", "l1.mix.sink", "l3.mix.sink", "l0.mix.b", "l0.mix.A_log",
                                  "l0.mix.dt_bias", "l0.mix.norm", "l0.mix.a2", "l2.mix.g2", "l0.mix.k.conv"])
def test_missing_weights_show(drop):
    W, toks = U.weights(MIX, 1), U.tokens(MIX[0], 60, 2)
    V = dict(W)
    V[drop] = np.full_like(W[drop], 1.0 if drop.endswith("mix.norm") or drop.endswith((".q.norm", ".k.norm")) else 0.0)
    assert U.rel_err(D.run(MIX[0], V, toks), D.run(MIX[0], W, toks)) > 20 * U.REL["float32"]


@pytest.mark.parametrize("key,value", [(("embedding", "scale"), 2.6), (("residual_mult",), 0.85), (("logit_softcap",), 1e6), (("norm", "eps"), 0.1)])
def test_constants_show(key, value):
    W, toks = U.weights(MIX, 1), U.tokens(MIX[0], 40, 2)
    cfg = json.loads(json.dumps(MIX[0]))
    at = cfg
    for k in key[:-1]:
        at = at[k]
    at[key[-1]] = value
    assert U.rel_err(D.run(cfg, W, toks), D.run(MIX[0], W, toks)) > 20 * U.REL["float32"]


def test_rotation_frequencies():
    sc = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 64}
    f, g = D.rotation_frequencies(5000.0, 12), D.rotation_frequencies(5000.0, 12, sc)
    wave = 2 * np.pi / f
    assert wave[0] < 16 and g[0] == f[0]
    assert wave[-1] > 64 and np.allclose(g[-1], f[-1] / 8)
    between = (wave > 16) & (wave < 64)
    assert between.any() and (g[between] < f[between]).all() and (g[between] > f[between] / 8).all()


def test_the_standout_key_is_seen_inside_the_window_only():
    case, W = U.standout()
    for dist in U.DISTANCES:
        for at in (0, 64):
            toks = U.standout_tokens(case, at, dist)
            want = D.run(case[0], W, toks)[-1:]
            hidden = toks.copy()
            hidden[at] = 5
            d = U.rel_err(D.run(case[0], W, hidden)[-1:], want)
            assert d > 3 * U.REL["bfloat16"] if dist < U.WINDOW else d < 1e-9, (dist, at, d)
    # the sink's share is seen, too
    V = dict(W, **{"l0.mix.sink": W["l0.mix.sink"] - 10})
    toks = U.standout_tokens(case, 0, 70)
    assert U.rel_err(D.run(case[0], V, toks)[-1:], D.run(case[0], W, toks)[-1:]) > 2 * U.REL["bfloat16"]


def test_the_kept_write_matters_for_hundreds_of_tokens():
    case, W = U.keeping()
    for dist in (1, 30, 400):
        toks = U.standout_tokens(case, 3, dist)
        hidden = toks.copy()
        hidden[3] = 5
        assert U.rel_err(D.run(case[0], W, hidden)[-1:], D.run(case[0], W, toks)[-1:]) > 2 * U.REL["bfloat16"], dist


def create(text, shapes=None):
    L, out = vk.load_library(), C.c_void_p()
    head = json.dumps({k: {"shape": list(v)} for k, v in (shapes or {}).items()}).encode()
    st = L.vkl_model_create_config_shapes(None, text.encode(), head, 64, vk.FP32, C.byref(out))
    return st, L.vkl_last_error().decode()


def test_config_reader():
    for case in U.CASES.values():
        st, msg = create(json.dumps(case[0]), U.shapes(U.weights(case, 1)))
        assert st == 3 and "null device" in msg  # the config itself was taken
    shapes = U.shapes(U.weights(MIX, 1))

    def broken(change, sh=shapes):
        c = json.loads(json.dumps(MIX[0]))
        change(c)
        return create(json.dumps(c), sh)

    assert "l0.mix.a1" in broken(lambda c: None, {})[1]
    assert "l2.mix.g1" in broken(lambda c: None, {k: v for k, v in shapes.items() if k != "l2.mix.g1"})[1]
    assert "vdim" in broken(lambda c: c["layers"][1]["mixer"].pop("vdim"))[1]
    assert "scale" in broken(lambda c: c["layers"][1]["mixer"].pop("scale"))[1]
    assert "conv" in broken(lambda c: c["layers"][0]["mixer"].pop("conv"))[1]
    assert "window" in broken(lambda c: c["layers"][1]["mixer"]["mask"].update(size=0))[1]
    assert "factor" in broken(lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("factor"))[1]
    assert "residual_mult" in broken(lambda c: c.pop("residual_mult"))[1]
    assert broken(lambda c: c["layers"][0].update(type="other"))[0] == 12
    assert broken(lambda c: c["layers"][0]["mlp"].update(kind="other"))[0] == 12
    assert "null device" in broken(lambda c: c["layers"][1]["mixer"]["rot"].pop("scaling"))[1]
