"""Small random models of the layer-list decoder designs for the tests: their sizes, their weights, and what
compares a run with the plain implementation in oracle/decoder.py."""
import numpy as np

from oracle import decoder as D

# fp32 runs differ from the float64 oracle by summation order only; bf16 runs by the operands' 8 bits
REL = {"float32": 2e-5, "bfloat16": 4e-2}


def attn(heads=6, kv_heads=2, dim=24, scale=None, bias_max=50, coef=0.4, every=16):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "bias_max": bias_max,
            "scale": scale if scale is not None else dim ** -0.5, "q_temp": {"coef": coef, "every": every}}


def dense(ff=112, limit=1.5):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(ff=40, experts=5, top=2):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(layers, width=96, vocab=150, loop=None, logit_scale=1.5):
    return {"architecture": "Rumalorn", "vocab": vocab, "width": width, "logit_scale": logit_scale, "loop": loop,
            "norm": {"eps": 1e-6}, "layers": [{"type": "attention", "mixer": a, "mlp": f} for a, f in layers]}


def weights(cfg, seed, rel_rows=20):
    """Random weights (as a checkpoint stores them) with scores of a few units, biases that matter and gates away from 1/2."""
    r = np.random.default_rng(seed)
    n = lambda std, *shape: r.normal(0, std, shape).astype(np.float32)
    W, V = cfg["width"], cfg["vocab"]
    w = {"embed": n(1.0, V, W), "head": n(W ** -0.5, V, W)}

    def norm(name):
        w[name], w[name + ".b"], w[name + ".alpha"] = 1 + n(0.3, W), n(0.2, W), np.float32(0.6 + 0.2 * r.random())

    norm("final.norm")
    if cfg["loop"]:
        w["loop.step"] = n(0.6, cfg["loop"]["times"], W)
    for i, layer in enumerate(cfg["layers"]):
        a, f, p = layer["mixer"], layer["mlp"], "l%d" % i
        H, G, d = a["heads"], a["kv_heads"], a["dim"]
        norm(p + ".norm1")
        p += ".mix"
        w[p + ".q"], w[p + ".q.b"] = n(1.8 * W ** -0.5, H * d, W), n(0.5, H * d)
        w[p + ".k"], w[p + ".k.b"] = n(1.8 * W ** -0.5, G * d, W), n(0.4, G * d)
        w[p + ".rel"] = n(1.2, rel_rows, H)
        w[p + ".g"] = n(2.0 * W ** -0.5, H, W)
        w[p + ".o"], w[p + ".o.b"] = n((H * d) ** -0.5, W, H * d), n(0.2, W)
        p = "l%d.mlp" % i
        if f and f["kind"] == "dense":
            for k, (o, c) in {"gate": (f["ff"], W), "up": (f["ff"], W), "down": (W, f["ff"])}.items():
                w["%s.%s" % (p, k)] = n((2.0 if k != "down" else 0.7) * c ** -0.5, o, c)
        elif f:
            E, top, ff = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"]
            for e in range(E):
                for k, (o, c) in {"gate": (ff, W), "up": (ff, W), "down": (W, ff)}.items():
                    w["%s.e%d.%s" % (p, e, k)] = n(1.5 * c ** -0.5, o, c)
            w[p + ".table"] = np.stack([r.permutation(E)[:top] for _ in range(V)]).astype(np.int32)
    return {k: (v if v.dtype.kind in "iu" else D.bf16_to_f32(D.f32_to_bf16(v)).reshape(v.shape)) for k, v in w.items()}


def tokens(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).astype(np.uint32)


def rel_err(got, want):
    """Worst row: RMS difference over the RMS of all wanted values."""
    d = np.asarray(got, np.float64) - want
    return float(np.sqrt((d ** 2).mean(-1)).max() / np.sqrt((np.asarray(want) ** 2).mean()))


# A model of each branch and several ways to combine them; no two share sizes.
CASES = {
    "attention only": config([(attn(), None)]),
    "dense": config([(attn(8, 4, 16), dense(72, 0.8))], width=80, vocab=97),
    "experts": config([(attn(4, 1, 32), moe(24, 3, 1))], width=64, vocab=77),
    "all experts": config([(attn(3, 3, 40), moe(36, 4, 4))], width=72, vocab=65),
    "loop from the first layer": config([(attn(2, 2, 20), dense(50)), (attn(10, 2, 36, bias_max=300), moe(28, 7, 3))], width=100, vocab=131,
                                        loop={"start": 0, "stop": 2, "times": 3}, logit_scale=0.7),
    "loop inside": config([(attn(6, 1, 8, bias_max=17, every=5), dense(40)), (attn(5, 5, 64), None), (attn(4, 2, 100, coef=-0.1), moe(20, 9, 2)), (attn(8, 2, 12), dense(200, 3.0))],
                          width=136, vocab=203, loop={"start": 1, "stop": 3, "times": 2}, logit_scale=2.5),
    "one pass": config([(attn(7, 7, 28), dense(60)), (attn(9, 3, 56), moe(52, 6, 2))], width=120, vocab=111, loop={"start": 1, "stop": 2, "times": 1}),
    "wide heads": config([(attn(2, 1, 200), dense(96)), (attn(3, 1, 144), None), (attn(4, 4, 256), moe(64, 2, 1))], width=192, vocab=90),
    "temperature and scale of 1": config([(attn(6, 3, 48, scale=0.05, coef=1.0, every=1), dense(88, 1.0))], width=112, vocab=140, logit_scale=1.0),
}


DISTANCES = (1, 7, 8, 9, 15, 16, 17, 62, 63, 64, 65, 127, 128, 129, 130, 131, 200, 330)


def standout(rows=16, far=130):
    """A model in which token 1 writes a key that token 2's query matches: their score stands out among all others,
    by enough to be seen among hundreds and by little enough that its distance's bias still counts."""
    cfg = config([(attn(2, 1, 32, scale=0.25, bias_max=far, coef=0.0), None)], width=64, vocab=40, logit_scale=1.0)
    W = weights(cfg, 51, rel_rows=rows)
    W["l0.mix.q"] *= 0.02
    W["l0.mix.k"] *= 0.3
    W["l0.mix.g"] *= 0.1
    W["l0.mix.o"] *= 3.0
    W["l0.norm1"][:2], W["l0.norm1.b"][:2], W["l0.norm1.alpha"] = 1, 0, np.float32(0.75)
    W["l0.mix.rel"] *= 0.6
    W["embed"][:, :2] = 0
    W["embed"][1, 0] = W["embed"][2, 1] = 4.0
    W["l0.mix.k"][5, 0] = 6.0                                  # token 1's key is long in column 5,
    W["l0.mix.q"][5, 1] = W["l0.mix.q"][32 + 5, 1] = 4.5       # and so is token 2's query, for both heads
    return cfg, {k: (v if v.dtype.kind in "iu" else D.bf16_to_f32(D.f32_to_bf16(v)).reshape(v.shape)) for k, v in W.items()}


def standout_tokens(cfg, at, dist):
    toks = tokens(cfg, at + dist + 1, dist) % 37 + 3
    toks[at], toks[-1] = 1, 2
    return toks
