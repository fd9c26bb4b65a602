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


def causal_attention(q, k, v, scale, bias=None):
    """q [T,H,d], k [T,G,d], v [T,G,e]; bias [distance, H] or None -> [T,H,e]."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]), q.dtype)
    back = np.arange(T)[:, None] - np.arange(T)[None, :]
    seen = back >= 0
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T) * scale
        if bias is not None:
            s = s + bias[np.maximum(back, 0), h]
        s = np.where(seen, s, -np.inf)
        p = np.exp(s - s.max(1, keepdims=True))
        out[:, h] = (p / p.sum(1, keepdims=True)) @ v[:, h // per]
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


def layer_runs(config):
    """(layer, pass) of every layer run in order; pass is None outside the loop."""
    n, lp = len(config["layers"]), config.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    return ([(i, None) for i in range(lp["start"])]
            + [(i, t) for t in range(lp["times"]) for i in range(lp["start"], lp["stop"])]
            + [(i, None) for i in range(lp["stop"], n)])


def run(config, weights, tokens, dtype=np.float64, layers_out=None, mixer=attention_mixer, ff=feed_forward):
    """Logits [T, vocab] of one sequence; the residual stream after every layer run is appended to layers_out."""
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
