"""Host side of the Petipel design (no GPU): the configuration reader accepts what the design allows and refuses the rest with a client
error, the registry keys on config.json's "architecture", and the float64 oracle the GPU tests lean on has the properties its mechanisms
are named for."""
import ctypes as C
import json
import math
import os

import numpy as np
import pytest

import petipel_oracle as P
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
    return P.make_config([P.hgrn2_layer(mlp=P.dense_ff()), P.attention_layer(mlp=P.moe_ff()), P.attention_layer(v_mix=False, q_temp=None), P.attention_layer(heads=6, dim=5)], width=40, vocab=77)


def test_config_reader_accepts_the_design(tmp_path):
    write_cfg(tmp_path, good_cfg())
    rc, info = model_info(tmp_path)
    assert rc == 0 and info["hidden"] == 40 and info["vocab"] == 77 and info["n_layers"] == 4
    assert model_info(tmp_path, dtype="float32")[0] == 0
    cfg = good_cfg()
    cfg["layers"][1]["mixer"].update(q_temp=None, v_mix=False)
    write_cfg(tmp_path, cfg)
    assert model_info(tmp_path)[0] == 0


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


@pytest.mark.parametrize("change", [
    mutate(["layers", 0, "type"], "gla"),
    mutate(["layers", 0, "mixer", "dim"], 0),
    mutate(["layers", 0, "mlp", "ff"], 0),
    mutate(["layers", 1, "mixer", "kv_heads"], 3),                     # does not divide heads
    mutate(["layers", 1, "mixer", "bias_max"], 0),
    drop(["layers", 1, "mixer", "bias_max"]),
    drop(["layers", 1, "mixer", "scale"]),
    mutate(["layers", 1, "mixer", "q_temp", "every"], 0),
    mutate(["layers", 3, "mixer", "vdim"], 10),                        # mixes values with a layer of another size
    mutate(["layers", 1, "mlp", "router", "top"], 7),                  # more than there are experts
    mutate(["layers", 1, "mlp", "expert", "limit"], 0.0),
    drop(["layers", 1, "mlp", "expert", "limit"]),
    mutate(["layers", 1, "mlp", "kind"], "sparse"),
    drop(["residual_mult"]),
    mutate(["vocab"], 0),
], ids=lambda f: "")
def test_config_reader_refuses(tmp_path, change):
    cfg = good_cfg()
    change(cfg)
    write_cfg(tmp_path, cfg)
    assert model_info(tmp_path)[0] == 400


def test_oracle_stack_is_causal():
    cfg = good_cfg()
    W = P.random_weights(cfg, 1)
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 60).tolist()
    assert np.abs(P.forward(cfg, W, toks[:17]) - P.forward(cfg, W, toks)[:17]).max() < 1e-9


def test_oracle_buckets():
    b = [P.bucket(n, 10, 40) for n in range(200)]
    assert b[:5] == [0, 1, 2, 3, 4] and b == sorted(b) and b[39] < 10 and set(b[40:]) == {9}
    # the logarithmic rows: row 5 + k starts at 5 (40 / 5)^(k / 5)
    assert [b.index(5 + k) for k in range(5)] == [math.ceil(5 * 8 ** (k / 5)) for k in range(5)]
    assert P.bucket(16, 16, 128) == 10 and P.bucket(15, 16, 128) == 9          # an exact power stands on its own row
    assert P.bucket(1, 2, 2) == 1 and P.bucket(0, 3, 9) == 0 and P.bucket(1, 3, 9) == 1


def test_oracle_attention_parts():
    assert P.query_temperature(0, 0.5, 4) == 1.0 and P.query_temperature(2, 0.5, 4) == 1.0 and np.isclose(P.query_temperature(3, 0.5, 4), 1.0 + 0.5 * math.log(2.0))
    q, k, v = (np.random.default_rng(s).standard_normal((6, 4)) for s in (3, 4, 5))
    out = P.biased_softmax_rows(q, k, v, 0.5, np.zeros(8), 30)
    assert np.allclose(out[0], v[0])
    assert np.allclose(P.biased_softmax_rows(q, k, v, 0.5, np.full(8, 3.0), 30), out)              # a constant bias changes nothing
    near = np.array([60.0, 0, 0, 0, 0, 0, 0, 0])
    assert np.allclose(P.biased_softmax_rows(q, k, v, 0.5, near, 30), v)                           # distance 0 alone
    assert np.allclose(P.biased_softmax_rows(q, k, v, 0.5, np.roll(near, 2), 30)[2:], v[:-2])      # distance 2 alone
    assert np.allclose(P.mixed_values(v, None, 0.3), v) and np.allclose(P.mixed_values(v, q, 1.0), q)
    assert np.allclose((P.unit_rms(v, 0.0) ** 2).mean(-1), 1.0)


def test_oracle_recurrence_and_feed_forward():
    rng = np.random.default_rng(6)
    q, v = rng.standard_normal((5, 3)), rng.standard_normal((5, 4))
    assert np.allclose(P.write_what_is_forgotten(q, np.zeros((5, 3)), v), q.sum(-1, keepdims=True) * v)       # nothing kept: every channel holds this token's value
    assert np.allclose(P.write_what_is_forgotten(q, np.ones((5, 3)), v), 0.0)                                 # nothing written
    f = P.forget_gate(np.array([-50.0, 0.0, 50.0]), 0.25)
    assert np.allclose(f, [0.25, 0.625, 1.0])
    z = rng.standard_normal((2, 9))
    assert np.allclose(P.poly_norm(z, (1.0, 0, 0, 0), 0.0), P.unit_rms(z, 0.0)) and np.allclose(P.poly_norm(z, (0, 0, 0, 0.7), 1e-5), 0.7)
    assert np.allclose(P.poly_norm(3.0 * z, (0.3, 0.5, -0.2, 0.1), 0.0), P.poly_norm(z, (0.3, 0.5, -0.2, 0.1), 0.0))          # only the direction counts
    one = {"e.gate": np.array([[100.0]]), "e.up": np.array([[100.0]]), "e.down": np.array([[1.0]])}
    assert np.allclose(P.expert(np.array([1.0]), one, "e.", 2.0), 2.0 * P.sigmoid(2 * 1.702) * 3.0)
    assert np.allclose(P.expert(np.array([-1.0]), one, "e.", 2.0), 0.0, atol=1e-6)
    idx, s = P.route(np.array([[1.0]]), np.array([[0.5], [-1.0], [2.0]]), 2)
    assert idx.tolist() == [[2, 0]] and np.allclose(s, P.sigmoid(np.array([[2.0, 0.5]])))
    assert np.allclose(P.norm(np.array([[3.0, 4.0]]), np.array([0.0, 1.0]), 0.0), np.array([[3.0, 8.0]]) / math.sqrt(12.5))
