"""Plain numpy restatement of the layer-list decoder designs (test infrastructure).

One function per mechanism, whole sequences at once, no cache, no batching, no kernel of the
library: what the CUDA path is compared with. Everything runs in the float type of its inputs
(float64 by default).
"""
import json
import math
import os
import struct

import numpy as np


# ---- checkpoint folder ---------------------------------------------------------------------
def bf16_to_f32(u16):
    return (np.asarray(u16, np.uint16).astype(np.uint32) << 16).view(np.float32)


def f32_to_bf16(x):
    """Nearest even."""
    u = np.ascontiguousarray(x, np.float32).view(np.uint32).astype(np.uint64)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def read_safetensors(path):
    """name -> array (bfloat16 widened to float32)."""
    raw = open(path, "rb").read()
    n = struct.unpack("<Q", raw[:8])[0]
    head = json.loads(raw[8:8 + n])
    out = {}
    for name, t in head.items():
        if name == "__metadata__":
            continue
        a, b = t["data_offsets"]
        buf = raw[8 + n + a:8 + n + b]
        if t["dtype"] == "BF16":
            v = bf16_to_f32(np.frombuffer(buf, np.uint16))
        else:
            v = np.frombuffer(buf, {"F32": np.float32, "I32": np.int32}[t["dtype"]])
        out[name] = v.reshape(t["shape"])
    return out


def write_safetensors(path, tensors):
    """Float arrays are stored as bfloat16, integer arrays as int32. Returns what was stored, widened."""
    head, blobs, at, back = {}, [], 0, {}
    for name, v in tensors.items():
        v = np.asarray(v)
        if v.dtype.kind in "iu":
            dt, data = "I32", v.astype("<i4").tobytes()
            back[name] = v.astype(np.int32)
        else:
            h = f32_to_bf16(v.reshape(-1))
            dt, data = "BF16", h.astype("<u2").tobytes()
            back[name] = bf16_to_f32(h).reshape(v.shape)
        head[name] = {"dtype": dt, "shape": list(v.shape), "data_offsets": [at, at + len(data)]}
        at += len(data)
        blobs.append(data)
    h = json.dumps(head).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))
    return back


def write_folder(path, config, tensors):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(config, f)
    return write_safetensors(os.path.join(path, "model.safetensors"), tensors)


# ---- mechanisms -----------------------------------------------------------------------------
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def linear(w, x, b=None):
    y = x @ w.T
    return y if b is None else y + b


def tanh_norm(x, w, b, alpha):
    """Dynamic Tanh: no statistics of x."""
    return np.tanh(alpha * x) * w + b


def query_temperature(pos, coef, every):
    return 1.0 + coef * np.log(np.floor((np.asarray(pos, np.float64) + 1) / every) + 1)


def distance_bucket(n, rows, far):
    """Row of the distance table for a key n positions back: the first half of the rows one by one, the
    rest on a logarithmic scale that ends at `far`. Whole-number arithmetic: row h + k starts where
    (n/h)^m >= (far/h)^k."""
    n, h = int(n), rows // 2
    if n < h:
        return n
    m, k = rows - h, 0
    while k < m and n ** m * h ** (k + 1) >= int(far) ** (k + 1) * h ** m:
        k += 1
    return min(rows - 1, h + k)


def distance_bias(table, far, n_max):
    """[n_max + 1, heads]: the bias at every distance."""
    return np.stack([table[distance_bucket(n, table.shape[0], far)] for n in range(n_max + 1)])


def causal_attention(q, k, v, scale, bias=None, window=None, sink=None):
    """q [T,H,d], k [T,G,d], v [T,G,e]; bias [distance, H] or None; window: keys a query sees, itself included, or
    None; sink [H] or None: one more term of each head's denominator, without a value -> [T,H,e]."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]), q.dtype)
    back = np.arange(T)[:, None] - np.arange(T)[None, :]
    seen = (back >= 0) & (back < window) if window else back >= 0
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T) * scale
        if bias is not None:
            s = s + bias[np.maximum(back, 0), h]
        s = np.where(seen, s, -np.inf)
        top = s.max(1, keepdims=True)
        if sink is not None:
            top = np.maximum(top, sink[h])
        p = np.exp(s - top)
        den = p.sum(1, keepdims=True)
        if sink is not None:
            den = den + np.exp(sink[h] - top)
        out[:, h] = (p / den) @ v[:, h // per]
    return out


def attention_mixer(h, W, p, mix, bias_of=distance_bias, temp_of=query_temperature):
    """Keys are the values; positions enter through the query's temperature and the distance bias only;
    one gate number per head."""
    T, H, G, d = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"]
    q = linear(W[p + ".q"], h, W[p + ".q.b"]).reshape(T, H, d)
    k = linear(W[p + ".k"], h, W[p + ".k.b"]).reshape(T, G, d)
    if mix.get("q_temp"):
        q = q * temp_of(np.arange(T), mix["q_temp"]["coef"], mix["q_temp"]["every"])[:, None, None].astype(h.dtype)
    bias = bias_of(W[p + ".rel"], mix["bias_max"], T - 1)
    o = causal_attention(q, k, k, mix["scale"], bias)
    o = o * sigmoid(linear(W[p + ".g"], h))[:, :, None]
    return linear(W[p + ".o"], o.reshape(T, H * d), W[p + ".o.b"])


def clamped_glu(h, W, p, limit):
    g = np.minimum(linear(W[p + ".gate"], h), limit)
    u = np.clip(linear(W[p + ".up"], h), -limit, limit)
    return linear(W[p + ".down"], g * sigmoid(1.702 * g) * (u + 1.0))


def silu_glu(h, W, p):
    z = linear(W[p + ".gate"], h)
    return linear(W[p + ".down"], z * sigmoid(z) * linear(W[p + ".up"], h))


def table_experts(h, W, p, tokens):
    """Each token id names its experts; equal weights."""
    table = W[p + ".table"]
    y = np.zeros_like(h)
    for t, tok in enumerate(tokens):
        for e in table[tok]:
            y[t] += silu_glu(h[t:t + 1], W, "%s.e%d" % (p, e))[0] / table.shape[1]
    return y


def feed_forward(h, W, p, mlp, tokens):
    if mlp["kind"] == "dense":
        return clamped_glu(h, W, p, mlp["limit"])
    return table_experts(h, W, p, tokens)


def rms(x, eps):
    """x over its root mean square."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def centred_rms_norm(x, w, eps):
    """The weight is stored as its difference from one."""
    return rms(x, eps) * (1.0 + w)


def rotation_frequencies(base, dims, scaling=None):
    """Angle per position of every pair; scaling stretches long wavelengths by a factor, short ones not at all, with
    a linear passage between original/high and original/low."""
    f = np.asarray(base, np.float64) ** (-np.arange(0, dims, 2) / dims)
    if not scaling:
        return f
    out = np.empty_like(f)
    for i, fi in enumerate(f):
        wave = 2 * math.pi / fi
        if wave < scaling["original"] / scaling["high"]:
            out[i] = fi
        elif wave > scaling["original"] / scaling["low"]:
            out[i] = fi / scaling["factor"]
        else:
            s = (scaling["original"] / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
            out[i] = (1 - s) * fi / scaling["factor"] + s * fi
    return out


def rotate_pairs(x, pos, freq):
    """x [T,H,d]: neighbours (2i, 2i+1) turn by pos * freq[i]; dimensions beyond the pairs stay."""
    n = 2 * len(freq)
    a = np.asarray(pos, np.float64)[:, None, None] * freq
    c, s = np.cos(a).astype(x.dtype), np.sin(a).astype(x.dtype)
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    y = x.copy()
    y[..., 0:n:2], y[..., 1:n:2] = u * c - v * s, v * c + u * s
    return y


def windowed_mixer(h, W, p, mix, eps, kv=None, attend=causal_attention, turn=rotate_pairs, freq_of=rotation_frequencies):
    """Norm over the whole query and key projection, rotation, a window and a sink per head. kv: the keys (after norm
    and rotation) and values of an earlier layer, which this one uses instead of its own. Returns output, keys, values."""
    T, H, G, d, e = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    freq, pos = freq_of(mix["rot"]["base"], mix["rot"]["dims"], mix["rot"].get("scaling")), np.arange(T)

    def side(name, heads):
        y = rms(linear(W["%s.%s" % (p, name)], h), eps) * W["%s.%s.norm" % (p, name)]
        return turn(y.reshape(T, heads, d), pos, freq)

    q = side("q", H)
    k, v = kv if kv is not None else (side("k", G), linear(W[p + ".v"], h).reshape(T, G, e))
    o = attend(q, k, v, mix["scale"], window=mix["mask"]["size"], sink=W[p + ".sink"])
    return linear(W[p + ".o"], o.reshape(T, H * e)), k, v


def silu(z):
    return z * sigmoid(z)


def short_convolution(x, taps):
    """x [T,C], taps [C,n]: causal, the last column is the current token's."""
    T, n = x.shape[0], taps.shape[1]
    y = np.zeros_like(x)
    for j in range(n):
        back = n - 1 - j
        y[back:] += x[:T - back] * taps[:, j] if back else x * taps[:, j]
    return y


def unit(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def softplus(z):
    return np.logaddexp(0.0, z)


def delta_recurrence(q, k, v, g, beta, S=None):
    """q, k, g [T,H,d], v [T,H,e], beta [T,H]: one token after the other, the read-out after the write."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2]), q.dtype) if S is None else S
    out = np.zeros(v.shape, q.dtype)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hde,hd->he", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hde,hd->he", S, q[t])
    return out


def delta_mixer(h, W, p, mix, eps, conv=short_convolution, recur=delta_recurrence, unit_of=unit):
    """Gated delta rule with a decay per head and key channel."""
    T, H, G, d, e = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    side = lambda n: silu(conv(linear(W["%s.%s" % (p, n)], h), W["%s.%s.conv" % (p, n)]))
    q = np.repeat(unit_of(side("q").reshape(T, G, d)) * d ** -0.5, H // G, 1)
    k = np.repeat(unit_of(side("k").reshape(T, G, d)), H // G, 1)
    v = side("v").reshape(T, H, e)
    beta = sigmoid(linear(W[p + ".b"], h))
    step = softplus(linear(W[p + ".a2"], linear(W[p + ".a1"], h)) + W[p + ".dt_bias"]).reshape(T, H, d)
    g = np.exp(-np.exp(W[p + ".A_log"])[:, None] * step)
    o = rms(recur(q, k, v, g, beta), eps) * W[p + ".norm"]
    o = o.reshape(T, H * e) * sigmoid(linear(W[p + ".g2"], linear(W[p + ".g1"], h)))
    return linear(W[p + ".o"], o)


def run_kupuzen(config, weights, tokens, dtype=np.float64, layers_out=None, attention=windowed_mixer, delta=delta_mixer, ff=silu_glu):
    """Both sublayers read the same stream through norms of their own; some attention layers read an earlier one's cache."""
    W = {k: v.astype(dtype) for k, v in weights.items()}
    eps, kvs = config["norm"]["eps"], {}
    x = W["embed"][np.asarray(tokens, np.int64)] * config["embedding"]["scale"]
    for i, L in enumerate(config["layers"]):
        p, mix = "l%d" % i, L["mixer"]
        h = centred_rms_norm(x, W[p + ".norm1"], eps)
        if L["type"] == "channel_delta":
            y = delta(h, W, p + ".mix", mix, eps)
        else:
            y, k, v = attention(h, W, p + ".mix", mix, eps, kvs.get(mix.get("kv_from")))
            kvs[i] = (k, v)
        if L["mlp"] is not None:
            y = y + ff(centred_rms_norm(x, W[p + ".norm2"], eps), W, p + ".mlp")
        x = x + config["residual_mult"] * y
        if layers_out is not None:
            layers_out.append(x.copy())
    y = linear(W["head"], centred_rms_norm(x, W["final.norm"], eps))
    cap = config["logit_softcap"]
    return cap * np.tanh(y / cap)


def layer_runs(config):
    """(layer, pass) of every layer run in order; pass is None outside the loop."""
    n, lp = len(config["layers"]), config.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    return ([(i, None) for i in range(lp["start"])]
            + [(i, t) for t in range(lp["times"]) for i in range(lp["start"], lp["stop"])]
            + [(i, None) for i in range(lp["stop"], n)])


def run(config, weights, tokens, dtype=np.float64, layers_out=None, **over):
    """Logits [T, vocab] of one sequence; the residual stream after every layer run is appended to layers_out. `over`
    replaces mechanisms of the design."""
    return {"Rumalorn": run_rumalorn, "Kupuzen": run_kupuzen}[config["architecture"]](config, weights, tokens, dtype, layers_out, **over)


def run_rumalorn(config, weights, tokens, dtype=np.float64, layers_out=None, mixer=attention_mixer, ff=feed_forward):
    W = {k: (v if v.dtype.kind in "iu" else v.astype(dtype)) for k, v in weights.items()}
    tokens = np.asarray(tokens, np.int64)
    emb = W["embed"][tokens]
    x = emb.copy()
    lp = config.get("loop")
    norm = lambda name, v: tanh_norm(v, W[name], W[name + ".b"], W[name + ".alpha"])
    for i, t in layer_runs(config):
        L, p = config["layers"][i], "l%d" % i
        if t is not None and i == lp["start"]:
            if t > 0:
                x = x + emb
            x = x + W["loop.step"][t]
        h = norm(p + ".norm1", x)
        y = mixer(h, W, p + ".mix", L["mixer"])
        if L["mlp"] is not None:
            y = y + ff(h, W, p + ".mlp", L["mlp"], tokens)
        x = x + y
        if layers_out is not None:
            layers_out.append(x.copy())
    return linear(W["head"], norm("final.norm", x)) * config["logit_scale"]
