"""The Petipel design of the hybrid family on the GPU against the slow float64 oracle (tests/petipel_oracle.py): each mechanism alone, and —
through Engine.trace_step, which drives the scheduler's own batch builder, pages and state slots — prompts cut into portions, token-by-token
decoding, mixed batches, pages and slots that are used again, far keys and the edges of the distance buckets, the steps of the query
temperature, the first tokens of a sequence, long decoding, the tensor-core kernels against the plain ones, and greedy generation through
the scheduler.  Small random checkpoints are written per test."""
import numpy as np
import pytest

import petipel_oracle as P

pytestmark = pytest.mark.gpu

F32_TOL = 2e-4          # fp32 engine against the float64 oracle (relative to the logits' spread)
BF16_TOL = 0.12         # bf16 matrices / activations: 90 % of the rows; the median is held to a quarter of it
SAME_TOL = 2e-5         # fp32 engine, two schedules of the same tokens


def engine(folder, dtype="float32", pages=8, slots=4, **kw):
    from opsagent_b200 import Engine
    return Engine(dict({"model_dir": str(folder), "dtype": dtype, "num_pages": pages, "max_seq_len": 64 * pages, "max_step_tokens": 64 * pages,
                        "max_batch": slots, "prefix_cache": 0}, **kw))


def checkpoint(tmp_path, cfg, seed=0, change=None, steady=False):
    W = P.random_weights(cfg, seed)
    if change:
        change(W)
    if steady:
        steady_routing(cfg, W)
    P.write_checkpoint(str(tmp_path), cfg, W)
    return W


def steady_routing(cfg, W):
    """bfloat16 rounding flips a near tie between two experts, and the row then answers with another expert.  Eight channels of the residual keep a code
    of the token (no sublayer writes there): its experts' logits differ by steps that rounding does not bridge."""
    rng = np.random.default_rng(77)
    W["embed"][:, :8] = P.bf16(np.stack([rng.permutation(np.linspace(-2.0, 2.0, 8)) for _ in range(cfg["vocab"])]))
    for name in W:
        if name.endswith(("mix.o", "down")):
            W[name][:8] = 0.0
        if name.endswith("norm2"):
            W[name][:8] = 0.0
        if name.endswith("router"):
            assert W[name].shape[0] <= 8
            W[name] = np.roll(np.eye(W[name].shape[0], W[name].shape[1]), int(name[1]), 0)


def scaled(suffixes, factor):
    def f(W):
        for name in W:
            if name.endswith(suffixes):
                W[name] = P.bf16(W[name] * factor)
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
    e = P.rel_err(got.astype(np.float64), want)
    if dtype == "float32":
        assert e.max() < F32_TOL, f"worst row {e.argmax()} differs by {e.max():.3e}"
    else:
        assert np.quantile(e, 0.9) < BF16_TOL and np.median(e) < BF16_TOL / 4, f"bf16 rows differ: median {np.median(e):.3e}, 90% {np.quantile(e, 0.9):.3e}"


A, H, D, M = P.attention_layer, P.hgrn2_layer, P.dense_ff, P.moe_ff
SINGLE = {
    "attention": [A()],
    "attention_plain_no_temperature_no_mixing": [A(q_temp=None, v_mix=False)],
    "attention_values_mixed_with_the_first_layer": [A(), A(heads=6, dim=6), A(heads=2, v_mix=False), A(rows=9, reach=17)],
    "attention_first_mixing_layer_is_not_the_first": [A(heads=3, kv_heads=3, vdim=5, v_mix=False), A(heads=2, kv_heads=1, vdim=7), A(heads=3, kv_heads=1, vdim=7, dim=3)],
    "attention_equal_heads_odd_sizes": [A(heads=3, kv_heads=3, dim=5, vdim=7, rows=11, reach=23, scale=0.9), A(heads=6, kv_heads=3, dim=1, vdim=7, rows=2, reach=2)],
    "attention_one_kv_head_temperature_every_token": [A(heads=6, kv_heads=1, dim=12, vdim=20, q_temp=(0.8, 1), reach=500, rows=32)],
    "attention_two_buckets_beyond_half": [A(rows=3, reach=60, scale=0.1), A(rows=12, reach=7)],
    "hgrn2": [H()],
    "hgrn2_one_head_one_channel": [H(heads=1, dim=1, vdim=3)],
    "hgrn2_sizes_off_every_vector": [H(heads=3, dim=6, vdim=7)],
    "hgrn2_rows_split_over_warps": [H(heads=2, dim=64, vdim=36)],
    "hgrn2_more_rows_than_registers_hold": [H(heads=1, dim=132, vdim=8)],
    "dense": [H(heads=1, mlp=D(64)), H(heads=1, mlp=D(50)), H(heads=1, mlp=D(9))],
    "experts_one_of_one": [H(heads=1, mlp=M(experts=1, top=1))],
    "experts_one_of_many": [H(heads=1, mlp=M(experts=7, top=1, ff=16))],
    "experts_three_small_limit": [A(mlp=M(experts=5, top=3, ff=20, limit=0.4))],
    "experts_all_chosen": [H(heads=1, mlp=M(experts=3, top=3, ff=9, limit=5.0))],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_each_mechanism_alone(tmp_path, name, dtype):
    odd = "odd" in name or "off" in name
    cfg = P.make_config(SINGLE[name], width=38 if odd else 40, eps=1e-6 if odd else 1e-5, mult=1.0 if odd else 0.6)
    W = checkpoint(tmp_path, cfg, seed=len(name), steady=dtype == "bfloat16")
    toks = tokens_of(cfg, 70, 1)                       # crosses a page border
    want = P.forward(cfg, W, toks)
    with engine(tmp_path, dtype) as eng:
        check(replay(eng, 1, toks, [70]), want, dtype)           # whole prompt
        check(replay(eng, 2, toks, [1, 1, 2, 3, 57, 2]), want, dtype)   # the first tokens alone, short portions, then token by token


def stack_cfg(**kw):
    layers = [H(mlp=D(48)), A(mlp=M()), A(heads=2, kv_heads=1, dim=16, vdim=6, reach=30, rows=8, q_temp=(0.7, 9), v_mix=False), H(heads=2, dim=12, vdim=8, mlp=M(experts=4, top=1, limit=0.8)),
              A(heads=6, kv_heads=2, dim=4, vdim=8, reach=90, rows=16, q_temp=None, mlp=D(56))]
    return P.make_config(layers, **kw)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_and_decoding_match_the_whole_prompt(tmp_path, dtype):
    cfg = stack_cfg()
    W = checkpoint(tmp_path, cfg, seed=3, steady=dtype == "bfloat16")
    toks = tokens_of(cfg, 140, 2)
    want = P.forward(cfg, W, toks)
    with engine(tmp_path, dtype) as eng:
        outs = [replay(eng, 7, toks, cuts) for cuts in ([140], [2, 62, 1, 2, 61, 12], [63, 2, 64], [5], [127, 1, 1, 11], [64, 64, 2, 2, 2, 2, 2, 2])]
    for got in outs:
        check(got, want, dtype)
        if dtype == "float32":
            assert P.rel_err(got.astype(np.float64), outs[0].astype(np.float64)).max() < SAME_TOL


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_requests_in_one_batch_and_reused_pages_and_slots(tmp_path, dtype):
    """Requests at different stages share every step (a prompt portion beside single tokens); later requests take over the pages and the state
    slots of finished ones: a stale cache row, a state that was not started from zero, or a wrong block table would show."""
    cfg = stack_cfg()
    W = checkpoint(tmp_path, cfg, seed=5, steady=dtype == "bfloat16")
    lens = {1: 100, 2: 37, 3: 66, 4: 90, 5: 20}
    toks = {r: tokens_of(cfg, n, 20 + r) for r, n in lens.items()}
    want = {r: P.forward(cfg, W, toks[r]) for r in lens}
    got = {r: [] for r in lens}
    at = {r: 0 for r in lens}
    with engine(tmp_path, dtype, pages=4, slots=2) as eng:
        def step(parts):
            entries, end = [], []
            for r, n in parts:
                n = min(n, lens[r] - at[r])
                entries.append((r, toks[r][at[r]:at[r] + n], list(range(n))))
                at[r] += n
                if at[r] == lens[r]:
                    end.append(r)
            out = eng.trace_step(entries, end)
            k = 0
            for r, t, w in entries:
                got[r].append(out[k:k + len(w)])
                k += len(w)
        step([(1, 60)])
        step([(1, 1), (2, 30)])                       # 1 decodes beside a portion of 2
        step([(1, 3), (2, 7)])                        # 2 ends: its page and slot are free
        step([(1, 36), (5, 2)])                       # 1 ends, 5 starts on 2's page and slot
        step([(5, 18), (3, 64)])                      # 5 ends; 3 fills exactly one page, in 1's slot
        step([(3, 2), (4, 2)])                        # 3 ends on a page's second token; 4 starts
        while at[4] < lens[4]:
            step([(4, 29)])
        assert eng.stats()["pages_free"] == 4
        for r in lens:                                # each alone, whole, in the same engine
            alone = replay(eng, 10 + r, toks[r], [lens[r]])
            e = P.rel_err(np.concatenate(got[r]).astype(np.float64), alone.astype(np.float64))
            assert e.max() < (SAME_TOL if dtype == "float32" else 3e-2)
    for r in lens:
        check(np.concatenate(got[r]), want[r], dtype)


def test_a_raised_bucket_decides_and_its_edges_count(tmp_path):
    """All bias rows but one are zero; the raised one owns the softmax wherever its distances exist.  The oracle with the bucket edges moved by
    one distance (the other readings of the table) differs at many rows by far more than the tolerance; the engine agrees with the right
    reading in prompts, in portions and in decoding, for a row below half, rows on the logarithmic scale and the last row (everything beyond)."""
    reach, rows, n = 77, 14, 230
    for raised in (3, 7, 10, 13):
        cfg = P.make_config([A(heads=4, kv_heads=2, dim=16, vdim=16, reach=reach, rows=rows, scale=0.2, q_temp=None)], width=32, vocab=50)
        W = P.random_weights(cfg, raised)
        W["l0.mix.rel"] = np.zeros((rows, 4))
        W["l0.mix.rel"][raised] = P.bf16(np.array([7.0, 6.0, 8.0, 7.5]))
        folder = tmp_path / str(raised)
        P.write_checkpoint(str(folder), cfg, W)
        toks = tokens_of(cfg, n, 40 + raised)
        want = P.forward(cfg, W, toks)
        true_bucket = P.bucket
        for shift in (-1, 1):
            try:
                P.bucket = lambda d, r, m: true_bucket(max(d + shift, 0), r, m)
                moved = P.forward(cfg, W, toks)
            finally:
                P.bucket = true_bucket
            assert (P.rel_err(moved, want) > 50 * F32_TOL).sum() > 40, "the bucket's edge does not show in the oracle"
        for dtype in ("float32", "bfloat16"):
            with engine(folder, dtype) as eng:
                for cuts in ([n], [70, 2, 3, 64, 61, 20], [30]):
                    got = replay(eng, 1, toks, cuts)
                    check(got, want, dtype)
                    if dtype == "bfloat16":
                        assert P.rel_err(got.astype(np.float64), want).max() < 0.1


def test_far_keys_decide(tmp_path):
    """Sharp queries and a bias that grows with the distance: single keys far back carry the rows.  Without its first page a prompt answers
    differently; the engine reads hundreds of tokens back, whole, in portions around page borders, and decoding."""
    cfg = P.make_config([H(heads=2), A(heads=2, kv_heads=1, dim=16, vdim=16, reach=150, rows=10, scale=1.0, q_temp=(0.5, 32)), A(heads=4, kv_heads=1, dim=16, vdim=16, reach=90, rows=20, scale=0.8)],
                        width=48, vocab=64)

    def sharpen(W):
        scaled(("mix.q",), 4.0)(W)
        for k in W:
            if k.endswith("rel"):
                W[k] = P.bf16(np.linspace(0.0, 5.0, W[k].shape[0])[:, None] + 0.3 * W[k])
    W = checkpoint(tmp_path, cfg, seed=9, change=sharpen)
    toks = tokens_of(cfg, 300, 5)
    want = P.forward(cfg, W, toks)
    assert np.median(P.rel_err(P.forward(cfg, W, toks[64:])[-100:], want[-100:])) > 100 * F32_TOL, "far keys do not show in the oracle"
    cuts = [63, 2, 62, 2, 1, 61, 2, 63, 30]
    with engine(tmp_path, pages=6) as eng:
        for c in ([300], cuts, [60]):
            check(replay(eng, 1, toks, c), want, "float32")
    with engine(tmp_path, "bfloat16", pages=6) as eng:
        for c in ([300], cuts, [60]):
            e = P.rel_err(replay(eng, 1, toks, c).astype(np.float64), want)
            assert np.quantile(e, 0.95) < 0.15, f"bf16, cuts {c}: 95% {np.quantile(e, 0.95):.3e}, worst {e.max():.3e}"


def test_query_temperature_steps(tmp_path):
    """The temperature changes right when (position + 1) reaches a multiple of `every`: the oracle with the step one position later differs at
    exactly those rows; the engine agrees with the right one, decoded over the step and in prompts."""
    every = 10
    cfg = P.make_config([A(heads=2, kv_heads=1, dim=16, vdim=16, scale=0.5, q_temp=(1.5, every))], width=32, vocab=40)
    W = checkpoint(tmp_path, cfg, seed=2, change=scaled(("mix.q",), 3.0))
    toks = tokens_of(cfg, 90, 3)
    want = P.forward(cfg, W, toks)
    true_t = P.query_temperature
    try:
        P.query_temperature = lambda p, c, e: true_t(p - 1, c, e)
        late = P.forward(cfg, W, toks)
    finally:
        P.query_temperature = true_t
    moved = np.flatnonzero(P.rel_err(late, want) > 5 * F32_TOL)
    assert len(moved) >= 6 and all((p + 1) % every == 0 for p in moved)
    for dtype in ("float32", "bfloat16"):
        with engine(tmp_path, dtype) as eng:
            for cuts in ([90], [9, 1, 1, 8, 2], [19, 2, 38, 2]):
                check(replay(eng, 1, toks, cuts), want, dtype)


def test_value_mixing_reads_the_same_token_of_the_first_mixing_layer(tmp_path):
    """Shares near one: the later layers' values are almost the first layer's.  Leaving the mixing out, mixing the other way round, or taking the layer
    before instead of the first each moves the oracle; the engine agrees, on pages another request has filled before."""
    cfg = P.make_config([A(v_mix=False), A(heads=2, kv_heads=2), A(), A(heads=6, dim=6)], width=40)

    def shares(W):
        for k in W:
            if k.endswith("vmix"):
                W[k] = P.bf16(np.array(0.85))
    W = checkpoint(tmp_path, cfg, seed=8, change=shares)
    toks, other = tokens_of(cfg, 80, 4), tokens_of(cfg, 100, 5)
    want = P.forward(cfg, W, toks)
    for lam in (0.0, 0.15):
        V = {k: (np.array(lam) if k.endswith("vmix") else v) for k, v in W.items()}
        assert np.median(P.rel_err(P.forward(cfg, V, toks), want)) > 50 * F32_TOL
    for dtype in ("float32", "bfloat16"):
        with engine(tmp_path, dtype, pages=2, slots=1) as eng:
            replay(eng, 1, other, [50, 2, 30])
            check(replay(eng, 2, toks, [33, 2, 2, 30]), want, dtype)


def test_a_forget_gate_near_one_keeps_the_first_tokens(tmp_path):
    """Gates within 1e-4 .. 1e-2 of one: the state remembers the whole sequence, and what a token writes (the gate's complement) is small, so the
    complement's own accuracy matters; gates at the lower bound forget at once.  Both in prompts, in portions and decoded."""
    cfg = P.make_config([H(heads=2, dim=16, vdim=16), H(heads=2, dim=16, vdim=16)], width=32, vocab=40)

    def gates(W):
        rng = np.random.default_rng(0)
        W["l0.mix.f.b"] = P.bf16(rng.uniform(4.0, 9.0, 32))
        W["l1.mix.f.b"] = P.bf16(rng.uniform(-12.0, -2.0, 32))
        W["l1.mix.lower"] = P.bf16(rng.uniform(0.0, 0.5, 32))
    W = checkpoint(tmp_path, cfg, seed=6, change=gates)
    toks = tokens_of(cfg, 200, 3)
    want = P.forward(cfg, W, toks)
    assert P.rel_err(P.forward(cfg, W, toks[10:])[-20:], want[-20:]).min() > 20 * F32_TOL          # the first ten tokens are still there at the end
    for dtype in ("float32", "bfloat16"):
        with engine(tmp_path, dtype) as eng:
            for cuts in ([200], [2, 63, 2, 2, 64, 40], [5]):
                check(replay(eng, 1, toks, cuts), want, dtype)


def test_router_weight_goes_into_the_expert(tmp_path):
    """Scores well below one and limits that bite: multiplying an expert's output instead of its input by the score, or renormalising the scores, moves
    the oracle; the engine agrees on the per-token path (few rows), the grouped path (many rows) and the plain path."""
    cfg = P.make_config([H(heads=1, mlp=M(experts=6, top=2, ff=32, limit=0.7)), A(mlp=M(experts=8, top=3, ff=16, limit=1.2))], width=40)
    W = checkpoint(tmp_path, cfg, seed=14, change=scaled((".gate", "mlp.e0.up", "mlp.e1.up"), 2.0), steady=True)
    toks = tokens_of(cfg, 90, 3)
    want = P.forward(cfg, W, toks)
    true_expert, true_route = P.expert, P.route
    try:
        P.route = lambda h, r, t: (true_route(h, r, t)[0], true_route(h, r, t)[1] / true_route(h, r, t)[1].sum(-1, keepdims=True))
        renormalised = P.forward(cfg, W, toks)
        P.route = lambda h, r, t: (true_route(h, r, t)[0], np.ones_like(true_route(h, r, t)[1]))
        unweighted = P.forward(cfg, W, toks)
    finally:
        P.expert, P.route = true_expert, true_route
    assert np.median(P.rel_err(renormalised, want)) > 50 * F32_TOL and np.median(P.rel_err(unweighted, want)) > 50 * F32_TOL
    with engine(tmp_path) as eng:
        check(replay(eng, 1, toks, [40, 2, 5]), want, "float32")
    for extra in ({}, {"hy_moe_grouped_rows": 1}, {"hy_moe_grouped_rows": 1000}, {"hy_tensor_core": 0}):
        with engine(tmp_path, "bfloat16", **extra) as eng:
            check(replay(eng, 1, toks, [40, 2, 5]), want, "bfloat16")


def test_first_tokens_start_from_nothing_on_a_reused_slot(tmp_path):
    cfg = stack_cfg()
    W = checkpoint(tmp_path, cfg, seed=4)
    X, Y = tokens_of(cfg, 30, 1), tokens_of(cfg, 9, 2)
    with engine(tmp_path, slots=1) as eng:
        check(replay(eng, 1, X, [30]), P.forward(cfg, W, X), "float32")
        check(replay(eng, 2, Y, [1, 1, 2]), P.forward(cfg, W, Y), "float32")          # the same slot, first tokens one by one
        check(replay(eng, 3, X, [2, 2]), P.forward(cfg, W, X), "float32")


def test_long_decoding(tmp_path):
    cfg = stack_cfg()
    W = checkpoint(tmp_path, cfg, seed=11)
    toks = tokens_of(cfg, 200, 7)
    with engine(tmp_path) as eng:
        check(replay(eng, 1, toks, [3]), P.forward(cfg, W, toks), "float32")     # 197 single-token steps over three page borders


TC_STACKS = {
    # sizes that take the tensor-core attention kernels: dim a multiple of 16, value heads of 16 .. 128 channels
    "buckets_inside_tiles": [A(heads=4, kv_heads=2, dim=32, vdim=48, reach=100, rows=32, mlp=D(96)), H(heads=2, dim=32, vdim=64, mlp=M(experts=8, top=2, ff=32)),
                             A(heads=8, kv_heads=2, dim=16, vdim=48, reach=400, rows=12, q_temp=(0.3, 100))],
    "large_group_and_wide_heads": [A(heads=20, kv_heads=1, dim=64, vdim=128, reach=600, rows=24, scale=0.1, q_temp=None), A(heads=6, kv_heads=1, dim=16, vdim=128, reach=30, rows=32, mlp=M(experts=5, top=1, ff=48)),
                                   H(heads=1, dim=128, vdim=96), H(heads=2, dim=96, vdim=24)],
    "one_head_per_group_and_other_widths": [A(heads=3, kv_heads=3, dim=48, vdim=80, reach=50, rows=7, mlp=D(64)), A(heads=2, kv_heads=2, dim=128, vdim=96, reach=64, rows=16, v_mix=False),
                                            H(heads=2, dim=40, vdim=88), H(heads=1, dim=16, vdim=128), A(heads=2, kv_heads=1, dim=16, vdim=32, v_mix=False), A(heads=2, kv_heads=1, dim=16, vdim=64, v_mix=False, reach=33)],
}


@pytest.mark.parametrize("name", sorted(TC_STACKS))
def test_bf16_tensor_core_path_and_plain_path_agree_with_the_oracle(tmp_path, name):
    """Prompts long enough for several query and key tiles, whole, in portions that straddle tiles and buckets, and decoding, on the tensor-core
    kernels and on the plain kernels (hy_tensor_core = 0)."""
    cfg = P.make_config(TC_STACKS[name], width=64, vocab=96)
    W = checkpoint(tmp_path, cfg, seed=13, change=scaled(("mix.q",), 1.5), steady=True)
    toks = tokens_of(cfg, 500, 8)
    want = P.forward(cfg, W, toks)
    for tc in (1, 0):
        with engine(tmp_path, "bfloat16", hy_tensor_core=tc) as eng:
            for cuts in ([500], [17, 33, 63, 130, 41, 180], [480]):
                e = P.rel_err(replay(eng, 1, toks, cuts).astype(np.float64), want)
                assert np.quantile(e, 0.95) < 0.1 and e.max() < 0.3, f"tensor cores {tc}, cuts {cuts}: 95% {np.quantile(e, 0.95):.3e}, worst {e.max():.3e}"


def test_greedy_generation_through_the_scheduler(tmp_path):
    """oa_tokens_submit -> continuous batching -> greedy sampling: three requests on two sequence slots (one waits), each compared with the
    oracle's greedy continuation wherever the oracle's top-1 margin is not a near tie."""
    cfg = stack_cfg()
    W = checkpoint(tmp_path, cfg, seed=12)
    prompts = [tokens_of(cfg, n, 30 + n) for n in (9, 70, 33)]
    n_new = 12
    with engine(tmp_path, pages=6, slots=2) as eng:
        tickets = [eng.tokens_submit(p, n_new, flags=1) for p in prompts]
        outs = [eng.wait(t).token_ids for t in tickets]
        assert eng.stats()["pages_free"] == 6
    for p, out in zip(prompts, outs):
        seq = list(p)
        assert len(out) == n_new
        for tok in out:
            lg = P.forward(cfg, W, seq)[-1]
            top2 = np.sort(lg)[-2:]
            if int(np.argmax(lg)) != tok:
                assert top2[1] - top2[0] < 1e-3, "greedy token differs from the oracle's outside a near tie"
                break
            seq.append(tok)
