"""Small random Kupuzen models for the tests: their sizes, their weights, and models in which one key, one sink or one
old write stands out."""
import numpy as np

from oracle import decoder as D
from decoder_util import REL, rel_err, tokens  # noqa: F401


def stored(W):
    """What a checkpoint keeps of the weights."""
    return {k: D.bf16_to_f32(D.f32_to_bf16(np.asarray(v).reshape(-1))).reshape(np.shape(v)) for k, v in W.items()}


def attn(heads=6, kv_heads=2, dim=24, vdim=40, window=21, rot=12, base=5000.0, scaling=(8.0, 1.0, 4.0, 64), scale=None, kv_from=None):
    mix = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
           "rot": {"base": base, "dims": rot}, "scale": scale if scale is not None else 1.3 * dim ** -0.5}
    if scaling:
        mix["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    if kv_from is not None:
        mix["kv_from"] = kv_from
    return "attention", mix


def delta(heads=4, kv_heads=2, dim=20, vdim=28, conv=3, ranks=(9, 14)):
    """ranks: of the decay's and the gate's two-step projections; they are in the tensors' shapes only."""
    return "channel_delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, ranks


def config(layers, width=96, vocab=150, embed=2.5, mult=0.6, cap=9.0, eps=1e-5):
    """layers: (mixer, feed-forward width or None). Returns the config and the layers' ranks."""
    cfg = {"architecture": "Kupuzen", "vocab": vocab, "width": width, "embedding": {"scale": embed}, "residual_mult": mult,
           "logit_softcap": cap, "norm": {"eps": eps},
           "layers": [{"type": m[0], "mixer": m[1], "mlp": {"kind": "dense", "ff": ff} if ff else None} for m, ff in layers]}
    return cfg, [m[2] if len(m) > 2 else None for m, _ in layers]


def weights(case, seed):
    """Random weights with scores of a few units, decays from a few tokens' memory to hundreds', gates away from 1/2."""
    cfg, ranks = case
    r = np.random.default_rng(seed)
    n = lambda std, *shape: r.normal(0, std, shape).astype(np.float32)
    W, V = cfg["width"], cfg["vocab"]
    w = {"embed": n(1.0, V, W), "head": n(4 * W ** -0.5, V, W), "final.norm": n(0.3, W)}
    for i, layer in enumerate(cfg["layers"]):
        a, p = layer["mixer"], "l%d.mix" % i
        H, G, d, e = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        w["l%d.norm1" % i] = n(0.3, W)
        if layer["type"] == "attention":
            w[p + ".q"], w[p + ".q.norm"] = n(W ** -0.5, H * d, W), 1 + n(0.3, H * d)
            if a.get("kv_from") is None:
                w[p + ".k"], w[p + ".k.norm"] = n(W ** -0.5, G * d, W), 1 + n(0.3, G * d)
                w[p + ".v"] = n(1.5 * W ** -0.5, G * e, W)
            w[p + ".sink"] = n(1.5, H)
        else:
            for k, c in (("q", G * d), ("k", G * d), ("v", H * e)):
                w["%s.%s" % (p, k)], w["%s.%s.conv" % (p, k)] = n(2 * W ** -0.5, c, W), n(0.7, c, a["conv"])
            w[p + ".b"] = n(2 * W ** -0.5, H, W)
            w[p + ".A_log"] = r.uniform(-4, 0, H).astype(np.float32)
            w[p + ".dt_bias"] = r.uniform(-3, 0, H * d).astype(np.float32)
            w[p + ".norm"] = 1 + n(0.3, e)
            for k, rows, rank in (("a", H * d, ranks[i][0]), ("g", H * e, ranks[i][1])):
                w["%s.%s1" % (p, k)], w["%s.%s2" % (p, k)] = n(W ** -0.5, rank, W), n(1.5 * rank ** -0.5, rows, rank)
        w[p + ".o"] = n((H * e) ** -0.5, W, H * e)
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            w["l%d.norm2" % i] = n(0.3, W)
            for k, (o, c) in {"gate": (ff, W), "up": (ff, W), "down": (W, ff)}.items():
                w["l%d.mlp.%s" % (i, k)] = n((1.5 if k != "down" else 0.7) * c ** -0.5, o, c)
    return stored(w)


def shapes(W):
    return {k: v.shape for k, v in W.items()}


# A model of each branch and several ways to combine them; no two share sizes.
CASES = {
    "attention only": config([(attn(), None)]),
    "attention and feed-forward": config([(attn(8, 4, 16, 16, 33, 16, scaling=None), 72)], width=80, vocab=97, embed=1.0, mult=1.0),
    "window of one": config([(attn(4, 1, 32, 24, 1, 2), 24)], width=64, vocab=77, mult=1.4),
    "window longer than the sequence": config([(attn(3, 3, 40, 72, 400, 40, 100.0, (2.0, 0.5, 8.0, 30)), 36)], width=72, vocab=65),
    "delta only": config([(delta(), None)], width=88, vocab=101),
    "delta, one head per key": config([(delta(3, 3, 32, 16, 1, (16, 16)), 52)], width=104, vocab=119, embed=0.5),
    "delta, many heads per key": config([(delta(6, 1, 48, 8, 2, (5, 70)), 60)], width=60, vocab=83, cap=30.0),
    "wide delta": config([(delta(2, 2, 200, 144, 5, (33, 3)), 40), (delta(2, 1, 256, 256, 4, (64, 65)), None)], width=112, vocab=90),
    "shared caches": config([(attn(4, 2, 28, 20, 17, 8), 40), (attn(4, 2, 28, 20, 5, 8, kv_from=0), None), (attn(4, 2, 28, 20, 90, 8, scale=0.4, kv_from=0), 64)],
                            width=68, vocab=140),
    "mixed": config([(delta(4, 2, 36, 20, 4, (12, 7)), 100), (attn(6, 3, 20, 36, 30, 10), 44), (delta(5, 5, 16, 64, 3, (8, 8)), None),
                     (attn(6, 3, 20, 36, 13, 10, kv_from=1), 80)], width=136, vocab=203, mult=0.8),
    "attention around delta": config([(attn(10, 2, 64, 48, 70, 32, 20000.0), 90), (delta(3, 1, 64, 96, 6, (20, 31)), 48), (attn(10, 2, 64, 48, 64, 32, 20000.0, kv_from=0), None),
                                      (attn(2, 1, 128, 200, 65, 64), 56)], width=120, vocab=111, eps=1e-3),
    "wide heads": config([(attn(2, 1, 208, 256, 40, 100), 96), (attn(5, 5, 144, 100, 129, 144, scaling=None), None)], width=192, vocab=94),
}


WINDOW = 66
DISTANCES = (1, 2, 15, 16, 17, 31, 32, 33, 62, 63, 64, 65, 66, 67, 68, 95, 128, 130)


def standout():
    """Windowed attention in which token 1 writes a key that token 2's query matches: its score stands out."""
    case = config([(attn(2, 1, 32, 32, WINDOW, 4, scaling=None, scale=0.35), None)], width=64, vocab=40, mult=1.0, embed=1.0, cap=50.0)
    W = weights(case, 51)
    W["l0.mix.q"] *= 0.05
    W["l0.mix.k"] *= 0.05
    W["l0.mix.q.norm"][:], W["l0.mix.k.norm"][:] = 1, 1
    W["l0.mix.o"] *= 3.0
    W["l0.mix.sink"][:] = 3.5
    W["l0.norm1"][:2] = 0
    W["embed"][:, :2] = 0
    W["embed"][1, 0] = W["embed"][2, 1] = 6.0
    W["l0.mix.k"][5, 0] = 3.0                                  # token 1's key is long in a dimension that does not turn,
    W["l0.mix.q"][5, 1] = W["l0.mix.q"][32 + 5, 1] = 3.0       # and so is token 2's query, for both heads
    return case, stored(W)


def standout_tokens(case, at, dist):
    toks = tokens(case[0], at + dist + 1, dist) % 37 + 3
    toks[at], toks[-1] = 1, 2
    return toks


def keeping():
    """A delta rule that forgets almost nothing and writes almost nothing, except for token 1; token 2 reads what token 1 wrote."""
    case = config([(delta(2, 1, 32, 32, 2, (4, 4)), None)], width=64, vocab=40, mult=1.0, embed=1.0, cap=50.0)
    W = weights(case, 53)
    for k in ("q", "k"):
        W["l0.mix." + k] *= 0.2
        W["l0.mix.%s.conv" % k][:] = [0.0, 1.0]
    W["l0.mix.A_log"][:] = -9.0
    W["l0.norm1"][:2] = 0
    W["embed"][:, :2] = 0
    W["embed"][1, 0] = W["embed"][2, 1] = 6.0
    W["l0.mix.b"][:, :] *= 0.05
    W["embed"][:, 2] = 3.0                                     # every token's step is small,
    W["l0.norm1"][2] = 0
    W["l0.mix.b"][:, 2] = -4.0
    W["l0.mix.b"][:, 0] = 6.0                                  # but for token 1's
    W["l0.mix.k"][7, 0] = W["l0.mix.q"][7, 1] = 6.0
    W["l0.mix.o"] *= 3.0
    return case, stored(W)
