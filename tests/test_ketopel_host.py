"""Host side of the Ketopel design (no GPU): the configuration reader accepts what the design allows and refuses the rest with a client
error, the registry keys on config.json's "architecture", and the float64 oracle the GPU tests lean on has the properties its mechanisms
are named for."""
import ctypes as C
import json
import math
import os

import numpy as np
import pytest

import ketopel_oracle as K
from opsagent_b200 import _lib


def model_info(folder, **extra):
    L = _lib.load()
    buf = C.create_string_buffer(4096)
    rc = L.oa_host_model_info(json.dumps(dict({"model_dir": str(folder)}, **extra)).encode(), buf, 4096)
    return rc, (json.loads(buf.value.decode()) if rc == 0 else None)


def write_cfg(folder, cfg):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)


def good_cfg():
    return K.make_config([K.delta_layer(mlp=K.dense_ff()), K.parallel_layer(mlp=K.dense_ff(30)), K.latent_layer(), K.parallel_layer(K.attention_part(scaling=None, softcap=None))],
                         width=40, vocab=77, loop=(1, 3, 3))


def test_config_reader_accepts_the_design(tmp_path):
    write_cfg(tmp_path, good_cfg())
    rc, info = model_info(tmp_path)
    assert rc == 0 and info["hidden"] == 40 and info["vocab"] == 77 and info["n_layers"] == 8        # executions: the looped layers count each pass
    assert model_info(tmp_path, dtype="float32")[0] == 0
    cfg = good_cfg()
    del cfg["loop"]
    cfg["layers"][1]["mixer"]["left"]["softcap"] = None
    cfg["layers"][1]["mixer"]["left"]["rot"]["scaling"] = None
    write_cfg(tmp_path, cfg)
    rc, info = model_info(tmp_path)
    assert rc == 0 and info["n_layers"] == 4


def mutate(path, value):
    def f(cfg):
        node = cfg
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
    return f


def drop(path):
    def f(cfg):
        node = cfg
        for k in path[:-1]:
            node = node[k]
        del node[path[-1]]
    return f


LEFT, RIGHT = ["layers", 1, "mixer", "left"], ["layers", 1, "mixer", "right"]


@pytest.mark.parametrize("change", [
    mutate(["layers", 0, "type"], "channel_delta"),
    mutate(["layers", 0, "type"], "attention"),
    mutate(["layers", 0, "mixer", "kv_heads"], 3),                     # does not divide heads
    mutate(["layers", 0, "mixer", "conv"], 0),
    mutate(["layers", 0, "mixer", "dim"], 0),
    mutate(["layers", 0, "mlp", "ff"], 0),
    mutate(["layers", 0, "mlp", "kind"], "moe"),
    mutate(LEFT + ["kv_heads"], 3),
    mutate(LEFT + ["rot", "dims"], 5),
    mutate(LEFT + ["rot", "dims"], 40),                                # more than a head has
    mutate(LEFT + ["rot", "scaling", "factor"], 0.0),
    drop(LEFT + ["rot", "scaling", "fast"]),
    drop(LEFT + ["scale"]),
    drop(RIGHT + ["decay"]),
    mutate(RIGHT + ["decay"], [0.5, 0.9]),                             # not one per head
    mutate(RIGHT + ["decay"], [0.5, 0.9, "x"]),
    drop(["layers", 1, "mixer", "left_scale"]),
    drop(["layers", 1, "mixer", "right_scale"]),
    mutate(["layers", 2, "mixer", "rot", "dims"], 6),                  # more than rot_dim
    drop(["layers", 2, "mixer", "kv_rank"]),
    mutate(["loop", "stop"], 1),
    mutate(["loop", "stop"], 5),
    mutate(["loop", "times"], 0),
    drop(["norm", "eps"]),
    mutate(["vocab"], 0),
], ids=lambda f: "")
def test_config_reader_refuses(tmp_path, change):
    cfg = good_cfg()
    change(cfg)
    write_cfg(tmp_path, cfg)
    assert model_info(tmp_path)[0] == 400


def test_oracle_stack_is_causal():
    cfg = good_cfg()
    W = K.random_weights(cfg, 1)
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 60).tolist()
    assert np.abs(K.forward(cfg, W, toks[:17]) - K.forward(cfg, W, toks)[:17]).max() < 1e-9


def test_oracle_schedule():
    assert K.schedule({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert K.schedule({"layers": [0] * 2}) == [(0, None), (1, None)]


def test_oracle_rotation():
    rng = np.random.default_rng(2)
    x = rng.standard_normal((9, 2, 10))
    rot = {"base": 100.0, "dims": 6}
    for inter in (False, True):
        y = K.rotate(x, rot, inter)
        assert np.allclose(y[0], x[0]) and np.allclose(y[..., 6:], x[..., 6:])
        assert np.allclose((y ** 2).sum(-1), (x ** 2).sum(-1))                                   # a rotation
        q, k = (np.repeat(v[None], 9, 0) for v in rng.standard_normal((2, 1, 10)))
        s = K.rotate(q, rot, inter)[:, 0] @ K.rotate(k, rot, inter)[:, 0].T
        assert np.isclose(s[5, 2], s[8, 5]) and np.isclose(s[3, 3], s[0, 0])                     # only the distance counts
    perm = [0, 2, 4, 1, 3, 5, 6, 7, 8, 9]                                                          # the two layouts are one rotation of reordered channels
    assert np.allclose(K.rotate(x, rot, True)[..., perm], K.rotate(x[..., perm], rot, False))
    f, amp = K.frequencies({"base": 100.0, "dims": 8, "scaling": {"factor": 4.0, "original": 50, "fast": 1000.0, "slow": 1e-3}})
    assert np.isclose(amp, 0.1 * math.log(4.0) + 1.0) and np.isclose(f[0], 1.0) and 0.25 < f[-1] * 100.0 ** 0.75 < 1.0 and all(np.diff(f) < 0)
    f, _ = K.frequencies({"base": 100.0, "dims": 8, "scaling": {"factor": 4.0, "original": 1e-4, "fast": 2.0, "slow": 2.0}})
    assert np.isclose(f[0], 1.0) and np.allclose(f[1:], [100.0 ** (-i / 4) / 4 for i in (1, 2, 3)])       # an empty ramp: every later pair is slowed by the whole factor


def test_oracle_recurrences():
    rng = np.random.default_rng(6)
    q, k, v = rng.standard_normal((5, 3)), rng.standard_normal((5, 3)), rng.standard_normal((5, 4))
    assert np.allclose(K.fading_memory(q, k, v, 0.0), (q * k).sum(-1, keepdims=True) * v)                       # nothing kept
    assert np.allclose(K.fading_memory(q, k, v, 1.0), np.tril(q @ k.T) @ v)                                     # everything kept
    one = np.ones(5)
    e = np.repeat(np.eye(3)[:1], 5, 0)
    assert np.allclose(K.corrected_memory(e, e, v, one, one), v)                                                # a key written again holds the last value only
    assert np.allclose(K.corrected_memory(q, k, v, one, 0 * one), 0.0)                                          # nothing written
    assert np.allclose(K.corrected_memory(q, np.eye(5)[:, :3], v, one, one), K.fading_memory(q, np.eye(5)[:, :3], v, 1.0))      # orthogonal keys need no correction
    x, taps = rng.standard_normal((4, 2)), rng.standard_normal((2, 3))
    y = K.short_convolution(x, taps)
    assert np.allclose(y[0], taps[:, 2] * x[0]) and np.allclose(y[3], taps[:, 0] * x[1] + taps[:, 1] * x[2] + taps[:, 2] * x[3])


def test_oracle_attention_and_feed_forward():
    v = np.random.default_rng(3).standard_normal((4, 2))
    assert np.allclose(K.causal_softmax(np.zeros((4, 4)), v), np.cumsum(v, 0) / np.arange(1, 5)[:, None])
    assert np.allclose(K.causal_softmax(np.eye(4)[[0, 0, 1, 2]] * 80.0, v)[1:], v[[0, 1, 2]])
    assert np.allclose(K.cap_scores(np.array([1e9, -1e9, 0.0]), 7.0), [7.0, -7.0, 0.0]) and K.cap_scores(5.0, None) == 5.0
    assert abs(K.gelu_tanh(1.0) - 0.8411920) < 1e-6 and K.gelu_tanh(0.0) == 0.0 and np.isclose(K.gelu_tanh(3.0) - K.gelu_tanh(-3.0), 3.0, atol=0.02)
    assert np.allclose(K.unit_rms(np.array([[3.0, 4.0]]), 0.0), np.array([[3.0, 4.0]]) / math.sqrt(12.5))
