"""The Ketopel design of the hybrid family on the GPU against the slow float64 oracle (tests/ketopel_oracle.py): each mechanism alone, and —
through Engine.trace_step, which drives the scheduler's own batch builder, pages and state slots — prompts cut into portions, token-by-token
decoding, mixed batches, pages and slots that are used again, far keys, what a looped block adds ahead of its passes, the soft cap, decays near
one and near zero, the first tokens of a sequence, long decoding, the tensor-core kernels against the plain ones, and greedy generation through
the scheduler.  Small random checkpoints are written per test."""
import numpy as np
import pytest

import ketopel_oracle as K

pytestmark = pytest.mark.gpu

F32_TOL = 2e-4          # fp32 engine against the float64 oracle (relative to the logits' spread)
BF16_TOL = 0.06         # bf16 matrices / activations: 90 % of the rows; the median is held to a third of it
SAME_TOL = 2e-5         # fp32 engine, two schedules of the same tokens


def engine(folder, dtype="float32", pages=8, slots=4, **kw):
    from opsagent_b200 import Engine
    return Engine(dict({"model_dir": str(folder), "dtype": dtype, "num_pages": pages, "max_seq_len": 64 * pages, "max_step_tokens": 64 * pages,
                        "max_batch": slots, "prefix_cache": 0}, **kw))


def checkpoint(tmp_path, cfg, seed=0, change=None):
    W = K.random_weights(cfg, seed)
    if change:
        change(W)
    K.write_checkpoint(str(tmp_path), cfg, W)
    return W


def scaled(suffixes, factor):
    def f(W):
        for name in W:
            if name.endswith(suffixes):
                W[name] = K.bf16(W[name] * factor)
    return f


def tokens_of(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def replay(eng, rid, toks, cuts):
    """feed toks to request rid in portions of the given sizes (the rest one by one), wanting every position; -> logits [len(toks), vocab]"""
    out, at = [], 0
    sizes = list(cuts)
    while at < len(toks):
        n = min(sizes.pop(0) if sizes else 1, len(toks) - at)
        out.append(eng.trace_step([(rid, toks[at:at + n], list(range(n)))], [rid] if at + n == len(toks) else []))
        at += n
    return np.concatenate(out)


def check(got, want, dtype):
    e = K.rel_err(got.astype(np.float64), want)
    if dtype == "float32":
        assert e.max() < F32_TOL, f"worst row {e.argmax()} differs by {e.max():.3e}"
    else:
        assert np.quantile(e, 0.9) < BF16_TOL and np.median(e) < BF16_TOL / 3, f"bf16 rows differ: median {np.median(e):.3e}, 90% {np.quantile(e, 0.9):.3e}"


A, R, P, L, D, F = K.attention_part, K.lightning_part, K.parallel_layer, K.latent_layer, K.delta_layer, K.dense_ff
SINGLE = {
    "parallel": [P()],
    "parallel_left_only_nearly": [P(A(heads=6, kv_heads=3, dim=6, vdim=7, dims=2, scaling=None), right_scale=0.01)],
    "parallel_right_only": [P(right=R(heads=2, dim=5, vdim=9, decay=[0.97, 0.4]), left_scale=0.0, right_scale=1.3)],
    "parallel_no_cap_no_scaling_all_rotated": [P(A(heads=3, kv_heads=3, dim=8, vdim=8, dims=8, scaling=None, softcap=None))],
    "parallel_nothing_rotated_negative_scale": [P(A(dims=0, scaling=None), left_scale=-0.8, right_scale=0.5)],
    "parallel_one_kv_head_odd_sizes": [P(A(heads=5, kv_heads=1, dim=11, vdim=5, dims=6, base=77.0, scaling=(2.0, 30, 3.0, 0.5), softcap=1.2), R(heads=1, dim=1, vdim=3, decay=[0.9]))],
    "parallel_steep_and_flat_scaling": [P(A(dim=16, dims=16, base=1e6, scaling=(8.0, 4096, 32.0, 1.0)), R(heads=2, dim=36, vdim=20)), P(A(dim=10, dims=10, base=20.0, scaling=(3.0, 8, 1.0, 1.0)))],
    "latent": [L()],
    "latent_odd_sizes": [L(heads=1, dim=5, rot_dim=2, vdim=3, kv_rank=7, base=50.0), L(heads=5, dim=1, rot_dim=6, vdim=9, kv_rank=20, scale=0.6)],
    "delta": [D()],
    "delta_equal_heads_two_taps": [D(heads=3, kv_heads=3, dim=6, vdim=7, conv=2)],
    "delta_one_key_head_one_tap": [D(heads=5, kv_heads=1, dim=4, vdim=4, conv=1)],
    "delta_one_channel_many_taps": [D(heads=1, kv_heads=1, dim=1, vdim=2, conv=9), D(heads=2, kv_heads=1, dim=9, vdim=5, conv=3)],
    "delta_rows_split_over_warps": [D(heads=2, kv_heads=1, dim=64, vdim=36)],
    "delta_more_rows_than_registers_hold": [D(heads=1, kv_heads=1, dim=132, vdim=8)],
    "feed_forward": [L(mlp=F(64)), D(mlp=F(50)), P(mlp=F(9)), L(mlp=F(1))],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_each_mechanism_alone(tmp_path, name, dtype):
    odd = "odd" in name or "one" in name
    cfg = K.make_config(SINGLE[name], width=38 if odd else 40, eps=1e-6 if odd else 1e-5, embed_scale=1.0 if odd else 1.7, loop=(0, 1, 1) if odd else None)
    W = checkpoint(tmp_path, cfg, seed=len(name))
    toks = tokens_of(cfg, 70, 1)                       # crosses a page border
    want = K.forward(cfg, W, toks)
    with engine(tmp_path, dtype) as eng:
        check(replay(eng, 1, toks, [70]), want, dtype)           # whole prompt
        check(replay(eng, 2, toks, [1, 1, 2, 3, 57, 2]), want, dtype)   # the first tokens alone, short portions, then token by token


def stack_cfg(loop=(1, 4, 3), **kw):
    layers = [L(mlp=F(48)), P(mlp=F(40)), D(heads=2, kv_heads=1, dim=12, vdim=8, conv=3), L(heads=2, dim=6, rot_dim=8, vdim=6, kv_rank=16), D(mlp=F(33)),
              P(A(heads=2, kv_heads=1, dim=16, vdim=6, dims=4, softcap=None), R(heads=2, dim=12, vdim=8), left_scale=1.3, right_scale=0.4)]
    return K.make_config(layers, loop=loop, **kw)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_and_decoding_match_the_whole_prompt(tmp_path, dtype):
    cfg = stack_cfg()
    W = checkpoint(tmp_path, cfg, seed=3)
    toks = tokens_of(cfg, 140, 2)
    want = K.forward(cfg, W, toks)
    with engine(tmp_path, dtype) as eng:
        outs = [replay(eng, 7, toks, cuts) for cuts in ([140], [2, 62, 1, 2, 61, 12], [63, 2, 64], [5], [127, 1, 1, 11], [64, 64, 2, 2, 2, 2, 2, 2])]
    for got in outs:
        check(got, want, dtype)
        if dtype == "float32":
            assert K.rel_err(got.astype(np.float64), outs[0].astype(np.float64)).max() < SAME_TOL


def run_crowd(eng, toks, plan):
    """plan: per step a list of (request, number of its next tokens); -> request -> logits of every position"""
    got, at = {r: [] for r in toks}, {r: 0 for r in toks}
    for parts in plan:
        entries, end = [], []
        for r, n in parts:
            n = min(n, len(toks[r]) - at[r])
            entries.append((r, toks[r][at[r]:at[r] + n], list(range(n))))
            at[r] += n
            if at[r] == len(toks[r]):
                end.append(r)
        out = eng.trace_step(entries, end)
        k = 0
        for r, t, w in entries:
            got[r].append(out[k:k + len(w)])
            k += len(w)
    assert all(at[r] == len(toks[r]) for r in toks)
    return {r: np.concatenate(g) for r, g in got.items()}


CROWD = [[(1, 60)], [(1, 1), (2, 30)], [(1, 3), (2, 7)],       # 1 decodes beside a portion of 2, which then ends: its page and slot are free
         [(1, 36), (5, 2)],                                    # 1 ends, 5 starts on 2's page and slot
         [(5, 18), (3, 64)],                                   # 5 ends; 3 fills exactly one page, in 1's slot
         [(3, 2), (4, 2)], [(4, 29)], [(4, 29)], [(4, 29)], [(4, 29)]]       # 3 ends on a page's second token


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_requests_in_one_batch_and_reused_pages_and_slots(tmp_path, dtype):
    """Requests at different stages share every step (a prompt portion beside single tokens); later requests take over the pages and the state
    slots of finished ones: a stale cache row, a state or a convolution tail that was not started from zero, or a wrong block table would show."""
    cfg = stack_cfg()
    W = checkpoint(tmp_path, cfg, seed=5)
    toks = {r: tokens_of(cfg, n, 20 + r) for r, n in {1: 100, 2: 37, 3: 66, 4: 90, 5: 20}.items()}
    with engine(tmp_path, dtype, pages=4, slots=2) as eng:
        got = run_crowd(eng, toks, CROWD)
        assert eng.stats()["pages_free"] == 4
        for r in toks:                                # each alone, whole, in the same engine
            alone = replay(eng, 10 + r, toks[r], [len(toks[r])])
            e = K.rel_err(got[r].astype(np.float64), alone.astype(np.float64))
            assert e.max() < (SAME_TOL if dtype == "float32" else 5e-2)
    for r in toks:
        check(got[r], K.forward(cfg, W, toks[r]), dtype)


@pytest.mark.parametrize("loop", [(0, 1, 4), (1, 3, 2), (3, 6, 2), (0, 6, 1), (5, 6, 3)])
def test_looped_block_adds_embedding_and_step(tmp_path, loop):
    """Where the block starts and ends, one pass or several.  Oracles that leave out the embedding, or take no or another pass's vector, differ by far
    more than the tolerance."""
    cfg = stack_cfg(loop=loop)
    W = checkpoint(tmp_path, cfg, seed=7, change=scaled(("loop.step",), 3.0))
    toks = tokens_of(cfg, 50, 4)
    want = K.forward(cfg, W, toks)
    for steps in ([np.zeros_like(W["loop.step"])] if loop[2] == 1 else [np.roll(W["loop.step"], 1, 0), np.zeros_like(W["loop.step"])]):
        assert np.median(K.rel_err(K.forward(cfg, dict(W, **{"loop.step": steps}), toks), want)) > 50 * F32_TOL
    true_schedule = K.schedule
    try:
        if loop[2] > 1:      # the embedding is left out
            K.schedule = lambda c: [(i, 0 if b else b) for i, b in true_schedule(c)]
            assert np.median(K.rel_err(K.forward(cfg, W, toks), want)) > 50 * F32_TOL
    finally:
        K.schedule = true_schedule
    with engine(tmp_path) as eng:
        for cuts in ([50], [20, 2, 7]):
            check(replay(eng, 1, toks, cuts), want, "float32")
    with engine(tmp_path, "bfloat16") as eng:
        check(replay(eng, 1, toks, [20, 2, 7]), want, "bfloat16")


def far_key_weights(W):
    """queries and keys so sharp that single keys own a row"""
    scaled(("left.q.norm", "left.k.norm"), 2.0)(W)
    for n in W:
        if n.endswith(("mix.q", "mix.uk")) and n[:3] in ("l1.", "l4."):
            W[n] = K.bf16(W[n] * 3.0)


def test_far_keys_decide(tmp_path):
    """Sharp queries: single keys far back carry the rows.  Without its first page a prompt answers differently; the engine reads hundreds of tokens
    back, whole, in portions around page borders, and decoding."""
    cfg = K.make_config([P(A(heads=4, kv_heads=2, dim=16, vdim=16, dims=6, scale=1.0, softcap=25.0)), L(heads=2, dim=16, rot_dim=16, vdim=16, kv_rank=64, scale=0.6), P(A(heads=2, kv_heads=1, dim=32, vdim=32, dims=32, scale=1.0, softcap=40.0))],
                        width=48, vocab=64)
    W = checkpoint(tmp_path, cfg, seed=9, change=far_key_weights)
    toks = tokens_of(cfg, 300, 5)
    want = K.forward(cfg, W, toks)
    assert np.median(K.rel_err(K.forward(cfg, W, toks[64:])[-100:], want[-100:])) > 100 * F32_TOL, "far keys do not show in the oracle"
    cuts = [63, 2, 62, 2, 1, 61, 2, 63, 30]
    with engine(tmp_path, pages=6) as eng:
        for c in ([300], cuts, [60]):
            check(replay(eng, 1, toks, c), want, "float32")
    with engine(tmp_path, "bfloat16", pages=6) as eng:
        for c in ([300], cuts, [60]):
            e = K.rel_err(replay(eng, 1, toks, c).astype(np.float64), want)
            assert np.quantile(e, 0.95) < 0.15, f"bf16, cuts {c}: 95% {np.quantile(e, 0.95):.3e}, worst {e.max():.3e}"


@pytest.mark.parametrize("kind", ["parallel", "latent"])
def test_one_planted_key_is_found_from_anywhere(tmp_path, kind):
    """One token's embedding points where every query looks: rows answer with its value wherever it stands — the first token, at a page border, hundreds
    back.  Dropping that one key moves the oracle; the engine agrees in prompts and decoding, for both kinds of attention."""
    layer = P(A(heads=2, kv_heads=1, dim=16, vdim=16, dims=0, scaling=None, scale=0.25, softcap=60.0), R(heads=1, dim=4, vdim=4), left_scale=1.0, right_scale=0.1) if kind == "parallel" else \
        L(heads=2, dim=16, rot_dim=2, vdim=16, kv_rank=32, scale=0.5)
    cfg = K.make_config([layer], width=32, vocab=40, embed_scale=1.0)

    def plant(W):
        W["embed"][:, 0] = 1.5                                   # every query sees channel 0
        W["embed"][39] = K.bf16(np.random.default_rng(5).standard_normal(32))
        W["embed"][:39, 1] = 0.0                                 # channel 1 marks the one token
        W["embed"][39, 1] = 6.0
        q, k = ("l0.mix.left.q", "l0.mix.left.k") if kind == "parallel" else ("l0.mix.q", "l0.mix.dkv")
        W[q][0] = 0.0
        W[q][0, 0] = 8.0
        W[k][0] = 0.0
        W[k][0, 1] = 8.0
        if kind == "latent":
            W["l0.mix.uk"][0] = 0.0
            W["l0.mix.uk"][0, 0] = 3.0
    W = checkpoint(tmp_path, cfg, seed=3, change=plant)
    for at in (0, 63, 64, 127):
        toks = [t % 39 for t in tokens_of(cfg, 260, at)]
        without = list(toks)
        toks[at] = 39
        want = K.forward(cfg, W, toks)
        assert np.median(K.rel_err(K.forward(cfg, W, without)[at + 1:], want[at + 1:])) > 0.1, "the planted key does not show in the oracle"
        for dtype in ("float32", "bfloat16"):
            with engine(tmp_path, dtype) as eng:
                for cuts in ([260], [at + 1, 2, 60], [30]):
                    check(replay(eng, 1, toks, cuts), want, dtype)


def test_soft_cap_bites(tmp_path):
    """Scores far beyond the cap: without it (or with a cap a tenth larger) the oracle differs; the engine agrees on the plain and the tensor-core kernels."""
    def capped(cap):
        return K.make_config([P(A(heads=4, kv_heads=2, dim=16, vdim=16, dims=8, scale=1.0, softcap=cap), left_scale=1.0, right_scale=0.2)], width=32, vocab=40)
    cfg = capped(3.0)
    W = checkpoint(tmp_path, cfg, seed=2, change=scaled(("left.q.norm",), 3.0))
    toks = tokens_of(cfg, 90, 3)
    want = K.forward(cfg, W, toks)
    for cap in (None, 3.3):
        assert np.median(K.rel_err(K.forward(capped(cap), W, toks), want)) > 20 * F32_TOL
    for dtype, extra in (("float32", {}), ("bfloat16", {}), ("bfloat16", {"hy_tensor_core": 0})):
        with engine(tmp_path, dtype, **extra) as eng:
            for cuts in ([90], [9, 1, 1, 8, 2], [19, 2, 38, 2]):
                check(replay(eng, 1, toks, cuts), want, dtype)


def decay_extremes(W):
    """the first layer keeps nearly everything, the third has a head that keeps nothing and one that keeps nearly everything"""
    W["l0.mix.A_log"][:] = K.bf16(np.array([-6.0, -7.0, -6.5, -5.0]))
    W["l2.mix.A_log"][:] = K.bf16(np.array([4.5, -6.0]))
    W["l2.mix.dt_bias"][:] = K.bf16(np.array([2.0, -1.0]))


def test_decays_near_one_and_near_zero(tmp_path):
    """Decays within 1e-3 of one: the state remembers the whole sequence; decays that underflow: it forgets at once.  In prompts, in portions and decoded."""
    cfg = K.make_config([D(heads=4, kv_heads=2, dim=16, vdim=16, conv=3), P(A(heads=2, kv_heads=1), R(heads=3, dim=16, vdim=24, decay=[0.9995, 0.5, 1e-3]), left_scale=0.1, right_scale=1.0),
                         D(heads=2, kv_heads=2, dim=24, vdim=32, conv=2)], width=32, vocab=40)
    W = checkpoint(tmp_path, cfg, seed=6, change=decay_extremes)
    toks = tokens_of(cfg, 200, 3)
    want = K.forward(cfg, W, toks)
    assert np.median(K.rel_err(K.forward(cfg, W, toks[10:])[-20:], want[-20:])) > 20 * F32_TOL          # the first ten tokens are still there at the end
    for dtype in ("float32", "bfloat16"):
        with engine(tmp_path, dtype) as eng:
            for cuts in ([200], [2, 63, 2, 2, 64, 40], [5], [33, 16, 17, 15, 31]):
                check(replay(eng, 1, toks, cuts), want, dtype)


def test_read_out_sees_the_write_and_keys_are_corrected(tmp_path):
    """Step sizes near one and the same few tokens over and over: what a key held is replaced.  An oracle without the correction, and one that reads
    before it writes, differ; the engine agrees."""
    cfg = K.make_config([D(heads=4, kv_heads=2, dim=16, vdim=16, conv=2)], width=32, vocab=6)

    def sure(W):
        W["l0.mix.b"] = K.bf16(np.abs(W["l0.mix.b"]) * 2.0)
        W["l0.mix.A_log"][:] = -4.0
        W["embed"] = K.bf16(np.abs(W["embed"]))
    W = checkpoint(tmp_path, cfg, seed=8, change=sure)
    toks = tokens_of(cfg, 120, 4)
    want = K.forward(cfg, W, toks)
    true_memory = K.corrected_memory
    try:
        K.corrected_memory = lambda q, k, v, g, b: K.fading_memory(q, k * b[:, None], v, 1.0)
        plain = K.forward(cfg, W, toks)
        K.corrected_memory = lambda q, k, v, g, b: np.concatenate([np.zeros((1, v.shape[1])), true_memory(np.roll(q, -1, 0), k, v, g, b)[:-1]])
        late = K.forward(cfg, W, toks)
    finally:
        K.corrected_memory = true_memory
    assert np.median(K.rel_err(plain, want)) > 50 * F32_TOL and np.median(K.rel_err(late, want)) > 50 * F32_TOL
    for dtype in ("float32", "bfloat16"):
        with engine(tmp_path, dtype) as eng:
            for cuts in ([120], [2, 30, 2, 50], [7]):
                check(replay(eng, 1, toks, cuts), want, dtype)


def test_first_tokens_start_from_nothing_on_a_reused_slot(tmp_path):
    cfg = stack_cfg()
    W = checkpoint(tmp_path, cfg, seed=4)
    X, Y = tokens_of(cfg, 30, 1), tokens_of(cfg, 9, 2)
    for dtype in ("float32", "bfloat16"):
        with engine(tmp_path, dtype, slots=1) as eng:
            check(replay(eng, 1, X, [30]), K.forward(cfg, W, X), dtype)
            check(replay(eng, 2, Y, [1, 1, 2]), K.forward(cfg, W, Y), dtype)          # the same slot, first tokens one by one
            check(replay(eng, 3, X, [2, 2]), K.forward(cfg, W, X), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(tmp_path, dtype):
    cfg = stack_cfg()
    W = checkpoint(tmp_path, cfg, seed=11)
    toks = tokens_of(cfg, 200, 7)
    with engine(tmp_path, dtype) as eng:
        check(replay(eng, 1, toks, [3]), K.forward(cfg, W, toks), dtype)     # 197 single-token steps over three page borders


TC_STACKS = {
    # sizes that take the tensor-core kernels of attention and of the recurrences
    "usual": [D(heads=4, kv_heads=2, dim=32, vdim=64, mlp=F(96)), P(A(heads=8, kv_heads=2, dim=64, vdim=64, dims=32), R(heads=2, dim=32, vdim=64)), L(heads=4, dim=32, rot_dim=16, vdim=48, kv_rank=64, mlp=F(80))],
    "wide_heads": [D(heads=2, kv_heads=1, dim=128, vdim=128, conv=3), P(A(heads=20, kv_heads=1, dim=128, vdim=128, dims=128), R(heads=2, dim=128, vdim=128)), L(heads=3, dim=96, rot_dim=32, vdim=112, kv_rank=128)],
    "other_widths": [D(heads=3, kv_heads=3, dim=48, vdim=80, conv=2), P(A(heads=3, kv_heads=3, dim=48, vdim=80, dims=16), R(heads=3, dim=40, vdim=88)), L(heads=5, dim=24, rot_dim=8, vdim=80, kv_rank=192),
                     D(heads=2, kv_heads=1, dim=16, vdim=16, conv=4), P(A(heads=2, kv_heads=2, dim=16, vdim=48, dims=2), R(heads=2, dim=16, vdim=24)), D(heads=2, kv_heads=2, dim=96, vdim=40)],
    "sizes_off_the_tiles": [D(heads=2, kv_heads=1, dim=20, vdim=36), P(A(heads=2, kv_heads=1, dim=24, vdim=40, dims=12), R(heads=2, dim=12, vdim=20)), L(heads=3, dim=12, rot_dim=4, vdim=20, kv_rank=40)],
}


@pytest.mark.parametrize("name", sorted(TC_STACKS))
def test_bf16_tensor_core_path_and_plain_path_agree_with_the_oracle(tmp_path, name):
    """Prompts long enough for several tiles and blocks, whole, in portions that straddle them, and decoding, on the tensor-core kernels and on the plain
    kernels (hy_tensor_core = 0)."""
    cfg = K.make_config(TC_STACKS[name], width=64, vocab=96, loop=(0, 2, 2))
    W = checkpoint(tmp_path, cfg, seed=13, change=scaled(("left.q.norm",), 1.5))
    toks = tokens_of(cfg, 640, 8)
    want = K.forward(cfg, W, toks)
    for tc in (1, 0):
        with engine(tmp_path, "bfloat16", pages=10, hy_tensor_core=tc) as eng:
            for cuts in ([640], [17, 33, 63, 130, 41, 3, 4, 5, 20, 280], [620]):
                e = K.rel_err(replay(eng, 1, toks, cuts).astype(np.float64), want)
                assert np.quantile(e, 0.95) < 0.05 and e.max() < 0.1, f"tensor cores {tc}, cuts {cuts}: 95% {np.quantile(e, 0.95):.3e}, worst {e.max():.3e}"


def test_bf16_crowd_on_the_tensor_core_kernels(tmp_path):
    """Portions beside single tokens through the kernels that have a form for each, with the extreme decays."""
    cfg = K.make_config([D(heads=4, kv_heads=2, dim=32, vdim=32, conv=3), P(A(heads=4, kv_heads=2, dim=32, vdim=32, dims=16), R(heads=3, dim=32, vdim=48, decay=[0.9995, 0.5, 1e-3])),
                         D(heads=2, kv_heads=2, dim=64, vdim=32), L(heads=2, dim=16, rot_dim=16, vdim=32, kv_rank=64)], width=64, vocab=80)
    W = checkpoint(tmp_path, cfg, seed=15, change=decay_extremes)
    toks = {r: tokens_of(cfg, n, 40 + r) for r, n in {1: 100, 2: 37, 3: 66, 4: 90, 5: 20}.items()}
    with engine(tmp_path, "bfloat16", pages=4, slots=2) as eng:
        got = run_crowd(eng, toks, CROWD)
    for r in toks:
        e = K.rel_err(got[r].astype(np.float64), K.forward(cfg, W, toks[r]))
        assert np.quantile(e, 0.95) < 0.05 and e.max() < 0.1, f"request {r}: 95% {np.quantile(e, 0.95):.3e}, worst {e.max():.3e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_scheduler(tmp_path, dtype):
    """oa_tokens_submit -> continuous batching -> greedy sampling: three requests on two sequence slots (one waits), each compared with the
    oracle's greedy continuation wherever the oracle's top-1 margin is not a near tie."""
    cfg = stack_cfg()
    W = checkpoint(tmp_path, cfg, seed=12)
    prompts = [tokens_of(cfg, n, 30 + n) for n in (9, 70, 33)]
    n_new = 12
    with engine(tmp_path, dtype, pages=6, slots=2) as eng:
        tickets = [eng.tokens_submit(p, n_new, flags=1) for p in prompts]
        outs = [eng.wait(t).token_ids for t in tickets]
        assert eng.stats()["pages_free"] == 6
    for p, out in zip(prompts, outs):
        seq = list(p)
        assert len(out) == n_new
        for tok in out:
            lg = K.forward(cfg, W, seq)[-1]
            if int(np.argmax(lg)) != tok:
                assert lg.max() - lg[tok] < (1e-3 if dtype == "float32" else 0.2), "greedy token differs from the oracle's outside a near tie"
                break
            seq.append(tok)
