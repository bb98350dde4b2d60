"""Plain float64 restatement of the Petipel design, one function per mechanism, no cache and no batching: every function takes the whole
sequence [T, ...] and loops over positions where a mechanism looks back.  It shares nothing with the engine; the GPU tests compare the
engine's logits (whole prompts, portions, decoding, mixed batches) with `forward()` of this file.

Notation: h is a sublayer's input [T, W]; weights are stored [out, in] and applied as h @ W.T; `w` is a dict name -> float64 ndarray."""
import json
import math
import os
import struct

import numpy as np


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def norm(x, weight, eps):
    """RMS norm whose stored weight counts from zero"""
    return unit_rms(x, eps) * (1.0 + weight)


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


# ---- attention ----------------------------------------------------------------------------------------------------------------------

def bucket(n, rows, reach):
    """row of the bias table for a distance n: one row per distance below rows / 2, then rows on a logarithmic scale up to `reach`, the last row beyond"""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + int(math.floor(math.log(n / half) / math.log(reach / half) * (rows - half) + 1e-9)))


def query_temperature(p, coef, every):
    return 1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0)


def biased_softmax_rows(q, k, v, scale, column, reach):
    """q, k [T, D], v [T, VD] of one head; column = the head's column of the bias table: position i sees j <= i, score scale q . k + bias of the distance"""
    T = q.shape[0]
    bias = np.array([column[bucket(n, len(column), reach)] for n in range(T)])
    out = np.zeros((T, v.shape[1]))
    for i in range(T):
        s = (k[: i + 1] @ q[i]) * scale + bias[i::-1]
        e = np.exp(s - s.max())
        out[i] = (e @ v[: i + 1]) / e.sum()
    return out


def mixed_values(v, first, lam):
    return v if first is None else (1.0 - lam) * v + lam * first


def attention(h, w, p, m, eps, carry):
    """carry: dict that hands the first value-mixing layer's values to the later ones"""
    T = h.shape[0]
    H, G, D, VD = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, D)
    k = (h @ w[p + "k"].T).reshape(T, G, D)
    v = unit_rms((h @ w[p + "v"].T).reshape(T, G, VD), eps)
    qt = m.get("q_temp")
    if qt:
        q = q * np.array([query_temperature(t, qt["coef"], qt["every"]) for t in range(T)])[:, None, None]
    if m.get("v_mix"):
        if "first" in carry:
            v = mixed_values(v, carry["first"], float(w[p + "vmix"]))
        else:
            carry["first"] = v
    gate = sigmoid(h @ w[p + "g"].T)
    out = np.zeros((T, H, VD))
    for hd in range(H):
        g = hd // (H // G)
        out[:, hd] = biased_softmax_rows(q[:, hd], k[:, g], v[:, g], m["scale"], w[p + "rel"][:, hd], m["bias_max"]) * gate[:, hd: hd + 1]
    return out.reshape(T, H * VD) @ w[p + "o"].T


# ---- gated recurrence -----------------------------------------------------------------------------------------------------------------

def forget_gate(z, lower):
    return lower + (1.0 - lower) * sigmoid(z)


def write_what_is_forgotten(q, f, v):
    """S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T, o_t = S_t^T q_t from S = 0; q, f [T, D], v [T, VD] of one head"""
    S = np.zeros((q.shape[1], v.shape[1]))
    out = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = f[t][:, None] * S + np.outer(1.0 - f[t], v[t])
        out[t] = S.T @ q[t]
    return out


def hgrn2(h, w, p, m, eps):
    T = h.shape[0]
    H, D, VD = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[p + "q"].T).reshape(T, H, D)
    f = forget_gate(h @ w[p + "f"].T + w[p + "f.b"], w[p + "lower"]).reshape(T, H, D)
    v = (h @ w[p + "v"].T).reshape(T, H, VD)
    o = np.stack([write_what_is_forgotten(q[:, i], f[:, i], v[:, i]) for i in range(H)], 1)
    return (unit_rms(o, eps) * w[p + "norm"]).reshape(T, H * VD) @ w[p + "o"].T


# ---- feed-forward -----------------------------------------------------------------------------------------------------------------------

def poly_norm(z, coef, eps):
    a, b, c, e = coef
    return a * unit_rms(z, eps) + b * unit_rms(z ** 2, eps) + c * unit_rms(z ** 3, eps) + e


def dense(h, w, p, eps):
    return poly_norm(h @ w[p + "up"].T, w[p + "act"], eps) @ w[p + "down"].T


def expert(x, w, p, limit):
    g = np.minimum(x @ w[p + "gate"].T, limit)
    u = np.clip(x @ w[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def route(h, router, top):
    """-> chosen experts [T, top] (largest score first) and their sigmoid scores"""
    z = h @ router.T
    idx = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    return idx, sigmoid(np.take_along_axis(z, idx, -1))


def experts(h, w, p, m):
    idx, s = route(h, w[p + "router"], m["router"]["top"])
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, sc in zip(idx[t], s[t]):
            y[t] += expert(sc * h[t], w, p + "e%d." % e, m["expert"]["limit"])
    return y


# ---- the stack ----------------------------------------------------------------------------------------------------------------------------

def forward(cfg, w, tokens, layers_out=None):
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][np.asarray(tokens)]
    carry = {}
    for i, l in enumerate(cfg["layers"]):
        p = "l%d." % i
        h = norm(x, w[p + "norm1"], eps)
        y = attention(h, w, p + "mix.", l["mixer"], eps, carry) if l["type"] == "attention" else hgrn2(h, w, p + "mix.", l["mixer"], eps)
        x = x + mult * norm(y, w[p + "norm1b"], eps)
        m = l.get("mlp")
        if m:
            h = norm(x, w[p + "norm2"], eps)
            y = dense(h, w, p + "mlp.", eps) if m["kind"] == "dense" else experts(h, w, p + "mlp.", m)
            x = x + mult * norm(y, w[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return norm(x, w["final.norm"], eps) @ w["head"].T


# ---- small random checkpoints for the tests ----------------------------------------------------------------------------------------

def attention_layer(heads=4, kv_heads=2, dim=8, vdim=8, reach=40, rows=12, q_temp=(0.4, 16), v_mix=True, scale=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "bias_max": reach, "scale": scale if scale is not None else dim ** -0.5}
    if q_temp:
        m["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    if v_mix:
        m["v_mix"] = True
    return {"type": "attention", "mixer": m, "mlp": mlp, "_rows": rows}


def hgrn2_layer(heads=3, dim=8, vdim=12, mlp=None):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": mlp}


def dense_ff(ff=48):
    return {"kind": "dense", "ff": ff}


def moe_ff(ff=24, experts=6, top=2, limit=1.5):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def make_config(layers, width=40, vocab=61, eps=1e-5, mult=0.6):
    return {"architecture": "Petipel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}


def tensor_shapes(cfg):
    W = cfg["width"]
    sh = {"embed": (cfg["vocab"], W), "head": (cfg["vocab"], W), "final.norm": (W,)}
    for i, l in enumerate(cfg["layers"]):
        p, m = "l%d." % i, l["mixer"]
        sh.update({p + "norm1": (W,), p + "norm1b": (W,)})
        H, D, VD = m["heads"], m["dim"], m["vdim"]
        if l["type"] == "attention":
            G = m["kv_heads"]
            sh.update({p + "mix.q": (H * D, W), p + "mix.k": (G * D, W), p + "mix.v": (G * VD, W), p + "mix.rel": (l.get("_rows", 12), H), p + "mix.g": (H, W), p + "mix.o": (W, H * VD)})
            if m.get("v_mix"):
                sh[p + "mix.vmix"] = ()
        else:
            sh.update({p + "mix.q": (H * D, W), p + "mix.f": (H * D, W), p + "mix.f.b": (H * D,), p + "mix.lower": (H * D,), p + "mix.v": (H * VD, W),
                       p + "mix.norm": (VD,), p + "mix.o": (W, H * VD)})
        ff = l.get("mlp")
        if not ff:
            continue
        sh.update({p + "norm2": (W,), p + "norm2b": (W,)})
        if ff["kind"] == "dense":
            sh.update({p + "mlp.up": (ff["ff"], W), p + "mlp.down": (W, ff["ff"]), p + "mlp.act": (4,)})
        else:
            F = ff["expert"]["ff"]
            sh[p + "mlp.router"] = (ff["router"]["experts"], W)
            for e in range(ff["router"]["experts"]):
                q = p + "mlp.e%d." % e
                sh.update({q + "gate": (F, W), q + "up": (F, W), q + "down": (W, F)})
    return sh


def bf16(a):
    """round to the nearest bfloat16 (ties to even), as float64"""
    b = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    b = ((b + 0x7FFF + ((b >> 16) & 1)) >> 16 << 16).astype(np.uint32)
    return b.view(np.float32).astype(np.float64).reshape(np.shape(a))


def random_weights(cfg, seed=0, spread=1.0):
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[1] if "." in name else name
        if last in ("norm1", "norm2", "norm1b", "norm2b") or name == "final.norm":
            v = 0.2 * rng.standard_normal(shape)
        elif last == "norm":
            v = 1.0 + 0.2 * rng.standard_normal(shape)
        elif last == "b":
            v = 1.5 + rng.standard_normal(shape)
        elif last == "lower":
            v = rng.uniform(0.0, 0.9, shape)
        elif last == "rel":
            v = 1.5 * rng.standard_normal(shape)
        elif last == "vmix":
            v = np.array(rng.uniform(0.2, 0.8))
        elif last == "act":
            v = rng.uniform(0.3, 1.0, shape) * np.array([1, -1, 1, 0.3])
        elif name == "embed":
            v = rng.standard_normal(shape)
        elif last == "router":
            v = 1.5 * rng.standard_normal(shape) / math.sqrt(shape[-1])
        else:
            v = spread * rng.standard_normal(shape) / math.sqrt(shape[-1])
        w[name] = bf16(v)
    return w


def write_checkpoint(folder, cfg, w):
    """config.json + model.safetensors (bfloat16): 8-byte header length, JSON header, data"""
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(dict(cfg, layers=[{k: v for k, v in l.items() if not k.startswith("_")} for l in cfg["layers"]]), f)
    header, blobs, at = {}, [], 0
    for name, a in w.items():
        raw = (np.ascontiguousarray(a, dtype=np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        header[name] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    hj = json.dumps(header).encode()
    hj += b" " * (-len(hj) % 8)
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(hj)) + hj + b"".join(blobs))


def rel_err(got, want):
    """per row: rms of the difference (means taken off) over the rms spread of the wanted logits"""
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt(((want - want.mean(-1, keepdims=True)) ** 2).mean())
