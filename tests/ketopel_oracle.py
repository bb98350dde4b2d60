"""Plain float64 restatement of the Ketopel design, one function per mechanism, no cache and no batching: every function takes the whole
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


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---- rotary positions -------------------------------------------------------------------------------------------------------------------

def frequencies(rot):
    """-> angular frequency of every pair and the amplitude of cos and sin"""
    n, base = rot["dims"], rot["base"]
    f = np.array([base ** (-2.0 * i / n) for i in range(n // 2)])
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def where(turns):
        return n * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(where(sc["fast"])), 0), min(math.ceil(where(sc["slow"])), n - 1)
    ramp = np.clip((np.arange(n // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, rot, interleaved):
    """x [T, heads, D]: the first rot.dims channels of every head turn by their position; the rest stays"""
    n = rot["dims"]
    f, amp = frequencies(rot)
    ang = np.arange(x.shape[0])[:, None] * f
    c, s = (np.cos(ang) * amp)[:, None], (np.sin(ang) * amp)[:, None]
    first = np.arange(0, n, 2) if interleaved else np.arange(n // 2)
    second = first + 1 if interleaved else first + n // 2
    y = x.copy()
    y[..., first] = x[..., first] * c - x[..., second] * s
    y[..., second] = x[..., second] * c + x[..., first] * s
    return y


# ---- softmax attention ------------------------------------------------------------------------------------------------------------------

def causal_softmax(score, v):
    """score [T, T] (row = query), v [T, VD]: position i weighs every j <= i"""
    out = np.zeros((score.shape[0], v.shape[1]))
    for i in range(score.shape[0]):
        e = np.exp(score[i, : i + 1] - score[i, : i + 1].max())
        out[i] = (e @ v[: i + 1]) / e.sum()
    return out


def cap_scores(s, cap):
    return cap * np.tanh(s / cap) if cap else s


def grouped_attention(h, w, p, m, eps):
    """capped causal attention, one norm over the whole query (key) projection, rotated halves"""
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (unit_rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]).reshape(T, H, D)
    k = (unit_rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]).reshape(T, G, D)
    v = (h @ w[p + "v"].T).reshape(T, G, m["vdim"])
    q, k = rotate(q, m["rot"], False), rotate(k, m["rot"], False)
    out = [causal_softmax(cap_scores(q[:, i] @ k[:, i // (H // G)].T * m["scale"], m.get("softcap")), v[:, i // (H // G)]) for i in range(H)]
    return np.concatenate(out, -1) @ w[p + "o"].T


def latent_attention(h, w, p, m, eps):
    """keys and values through a normed latent, one rotated key part shared by the heads, a sigmoid gate per head"""
    T, H, D, R, K = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).reshape(T, H, D + R)
    down = h @ w[p + "dkv"].T
    c = unit_rms(down[:, :K], eps) * w[p + "dkv.norm"]
    shared = rotate(down[:, None, K:], m["rot"], True)[:, 0]
    q_rot = rotate(q[..., D:], m["rot"], True)
    k = (c @ w[p + "uk"].T).reshape(T, H, D)
    v = (c @ w[p + "uv"].T).reshape(T, H, m["vdim"])
    gate = sigmoid(h @ w[p + "g"].T)
    out = [causal_softmax((q[:, i, :D] @ k[:, i].T + q_rot[:, i] @ shared.T) * m["scale"], v[:, i]) * gate[:, i: i + 1] for i in range(H)]
    return np.concatenate(out, -1) @ w[p + "o"].T


# ---- recurrences ------------------------------------------------------------------------------------------------------------------------

def fading_memory(q, k, v, decay):
    """S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t from S = 0, of one head"""
    S = np.zeros((q.shape[1], v.shape[1]))
    out = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = decay * S + np.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out


def lightning(h, w, p, m, eps):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    q, k = (silu(h @ w[p + n].T).reshape(T, H, D) for n in "qk")
    v = silu(h @ w[p + "v"].T).reshape(T, H, m["vdim"])
    o = np.concatenate([fading_memory(q[:, i], k[:, i], v[:, i], m["decay"][i]) for i in range(H)], -1)
    return (unit_rms(o, eps) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def side_by_side(h, w, p, m, eps):
    return m["left_scale"] * grouped_attention(h, w, p + "left.", m["left"], eps) + m["right_scale"] * lightning(h, w, p + "right.", m["right"], eps)


def short_convolution(x, taps):
    """x [T, C], taps [C, n]: the last tap weighs the current row, rows before the first are zero"""
    n = taps.shape[1]
    padded = np.concatenate([np.zeros((n - 1, x.shape[1])), x])
    return sum(padded[j: j + x.shape[0]] * taps[:, j] for j in range(n))


def unit_vector(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def corrected_memory(q, k, v, g, beta):
    """S <- g_t S; u = beta_t (v_t - S^T k_t); S <- S + k_t u^T; o_t = S^T q_t, of one head"""
    S = np.zeros((q.shape[1], v.shape[1]))
    out = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = g[t] * S
        S = S + np.outer(k[t], beta[t] * (v[t] - S.T @ k[t]))
        out[t] = S.T @ q[t]
    return out


def gated_delta(h, w, p, m, eps):
    T, H, G, D, VD = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_convolution(h @ w[p + n].T, w[p + n + ".conv"])) for n in "qkv")
    q = unit_vector(q.reshape(T, G, D)) * D ** -0.5
    k = unit_vector(k.reshape(T, G, D))
    v = v.reshape(T, H, VD)
    beta = sigmoid(h @ w[p + "b"].T)
    g = np.exp(-np.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = np.stack([corrected_memory(q[:, i // (H // G)], k[:, i // (H // G)], v[:, i], g[:, i], beta[:, i]) for i in range(H)], 1)
    o = unit_rms(o, eps) * w[p + "norm"] * silu(h @ w[p + "g"].T).reshape(T, H, VD)
    return o.reshape(T, H * VD) @ w[p + "o"].T


# ---- the stack --------------------------------------------------------------------------------------------------------------------------

def dense(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


MIXERS = {"parallel": side_by_side, "latent_attention": latent_attention, "delta": gated_delta}


def schedule(cfg):
    """-> (layer, number of the pass that starts here or None) per execution"""
    lp, out, i = cfg.get("loop"), [], 0
    while i < len(cfg["layers"]):
        if lp and i == lp["start"]:
            out += [(k, t if k == i else None) for t in range(lp["times"]) for k in range(i, lp["stop"])]
            i = lp["stop"]
        else:
            out.append((i, None))
            i += 1
    return out


def forward(cfg, w, tokens, layers_out=None):
    eps = cfg["norm"]["eps"]
    first = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    x = first
    for i, begins in schedule(cfg):
        if begins is not None:
            if begins > 0:
                x = x + first
            x = x + w["loop.step"][begins]
        l, p = cfg["layers"][i], "l%d." % i
        x = x + MIXERS[l["type"]](unit_rms(x, eps) * w[p + "norm1"], w, p + "mix.", l["mixer"], eps)
        if l.get("mlp"):
            x = x + dense(unit_rms(x, eps) * w[p + "norm2"], w, p + "mlp.")
        if layers_out is not None:
            layers_out.append(x.copy())
    return (unit_rms(x, eps) * w["final.norm"]) @ w["head"].T


# ---- small random checkpoints for the tests ---------------------------------------------------------------------------------------------

def dense_ff(ff=48):
    return {"kind": "dense", "ff": ff}


def attention_part(heads=4, kv_heads=2, dim=12, vdim=10, dims=8, base=500.0, scaling=(4.0, 64, 8.0, 1.0), scale=None, softcap=5.0):
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot, "scale": scale if scale is not None else dim ** -0.5}
    if softcap:
        m["softcap"] = softcap
    return m


def lightning_part(heads=3, dim=8, vdim=12, decay=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [1.0 - 2.0 ** -(1 + 2 * h) for h in range(heads)]}


def parallel_layer(left=None, right=None, left_scale=0.7, right_scale=1.4, mlp=None):
    return {"type": "parallel", "mixer": {"left": left or attention_part(), "right": right or lightning_part(), "left_scale": left_scale, "right_scale": right_scale}, "mlp": mlp}


def latent_layer(heads=3, dim=8, rot_dim=4, vdim=10, kv_rank=12, base=300.0, scale=None, mlp=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": {"base": base, "dims": rot_dim},
                                                  "scale": scale if scale is not None else (dim + rot_dim) ** -0.5}, "mlp": mlp}


def delta_layer(heads=4, kv_heads=2, dim=8, vdim=12, conv=4, mlp=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def make_config(layers, width=40, vocab=61, eps=1e-5, embed_scale=1.7, loop=None):
    cfg = {"architecture": "Ketopel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed_scale}, "layers": layers}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def tensor_shapes(cfg):
    W = cfg["width"]
    sh = {"embed": (cfg["vocab"], W), "head": (cfg["vocab"], W), "final.norm": (W,)}
    if cfg.get("loop"):
        sh["loop.step"] = (cfg["loop"]["times"], W)
    for i, l in enumerate(cfg["layers"]):
        p, m = "l%d." % i, l["mixer"]
        x = p + "mix."
        sh[p + "norm1"] = (W,)
        if l["type"] == "parallel":
            a, b = m["left"], m["right"]
            H, G, D, VD = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            y = x + "left."
            sh.update({y + "q": (H * D, W), y + "k": (G * D, W), y + "v": (G * VD, W), y + "q.norm": (H * D,), y + "k.norm": (G * D,), y + "o": (W, H * VD)})
            H, D, VD = b["heads"], b["dim"], b["vdim"]
            y = x + "right."
            sh.update({y + "q": (H * D, W), y + "k": (H * D, W), y + "v": (H * VD, W), y + "g": (H * VD, W), y + "o": (W, H * VD), y + "norm": (H * VD,)})
        elif l["type"] == "latent_attention":
            H, D, R, VD, K = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            sh.update({x + "q": (H * (D + R), W), x + "dkv": (K + R, W), x + "dkv.norm": (K,), x + "uk": (H * D, K), x + "uv": (H * VD, K), x + "g": (H, W), x + "o": (W, H * VD)})
        else:
            H, G, D, VD, n = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            sh.update({x + "q": (G * D, W), x + "q.conv": (G * D, n), x + "k": (G * D, W), x + "k.conv": (G * D, n), x + "v": (H * VD, W), x + "v.conv": (H * VD, n),
                       x + "b": (H, W), x + "A_log": (H,), x + "norm": (VD,), x + "a": (H, W), x + "dt_bias": (H,), x + "g": (H * VD, W), x + "o": (W, H * VD)})
        if l.get("mlp"):
            F = l["mlp"]["ff"]
            sh.update({p + "norm2": (W,), p + "mlp.gate": (F, W), p + "mlp.up": (F, W), p + "mlp.down": (W, F)})
    return sh


def bf16(a):
    """round to the nearest bfloat16 (ties to even), as float64"""
    b = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    b = ((b + 0x7FFF + ((b >> 16) & 1)) >> 16 << 16).astype(np.uint32)
    return b.view(np.float32).astype(np.float64).reshape(np.shape(a))


def random_weights(cfg, seed=0):
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[1] if "." in name else name
        if last in ("norm", "norm1", "norm2"):
            v = 1.0 + 0.2 * rng.standard_normal(shape)
        elif last == "conv":
            v = rng.standard_normal(shape) / math.sqrt(shape[-1])
        elif last == "A_log":
            v = rng.uniform(-1.5, 0.7, shape)
        elif last == "dt_bias":
            v = rng.uniform(-3.0, 0.5, shape)
        elif last == "step":
            v = 0.5 * rng.standard_normal(shape)
        elif name == "embed":
            v = rng.standard_normal(shape)
        else:
            v = rng.standard_normal(shape) / math.sqrt(shape[-1])
        w[name] = bf16(v)
    return w


def write_checkpoint(folder, cfg, w):
    """config.json + model.safetensors (bfloat16): 8-byte header length, JSON header, data"""
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
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
