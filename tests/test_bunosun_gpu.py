"""Bunosun on the GPU against the float64 oracle (tests/bunosun_oracle.py): small made-up configurations with random or hand-made
weights.  Covered: each mechanism alone, the model layer by layer, prefill against token-by-token decoding, portions down to two
tokens, unequal batches, reuse of pages and slots, keys far back / at page borders / just inside and just outside a window (in
either map), state carried from far back, the convolution's inputs across cuts, the loop's passes, the router's groups, the first
tokens, long decoding, other sizes, the tensor-core paths of prompt passes, a model folder, and greedy generation through the
scheduler."""
import json

import numpy as np
import pytest

from distributed_inference_server_b200 import ContinuousBatcher, InferenceParams, models
from tests import _bunosun_util as U

pytestmark = pytest.mark.gpu
F32_TOL = 2e-5


def toks(n, vocab=53, seed=0):
    return [int(x) for x in np.random.default_rng(seed).integers(0, vocab, n)]


MECHANISMS = {
    "attention_alone": [(U.attention(), None)],
    "attention_whole_past": [(U.attention(window=0), None)],
    "attention_window_of_one": [(U.attention(window=1), None)],
    "attention_window_of_two": [(U.attention(window=2), None)],
    "attention_nothing_rotated": [(U.attention(rot=0), None)],
    "attention_every_coordinate_rotated_unscaled": [(U.attention(heads=3, kv_heads=1, dim=8, vdim=6, rot=8, factor=0), None)],
    "attention_strongly_scaled_frequencies": [(U.attention(dim=8, rot=8, base=30.0, factor=0.25), None)],
    "attention_no_difference_constant": [(U.attention(diff=0.0), None)],
    "attention_values_smaller_than_keys": [(U.attention(heads=2, kv_heads=2, dim=12, vdim=3, window=64), None)],
    "delta_alone": [(U.delta(), None)],
    "delta_one_tap": [(U.delta(conv=1), None)],
    "delta_two_taps_one_key_head": [(U.delta(heads=6, kv_heads=1, dim=6, vdim=5, conv=2), None)],
    "delta_four_taps_as_many_key_heads": [(U.delta(heads=3, kv_heads=3, dim=12, vdim=8, conv=4, decay_rank=8, gate_rank=16), None)],
    "delta_seven_taps": [(U.delta(conv=7, decay_rank=1, gate_rank=1), None)],
    "mixture_beside_attention": [(U.attention(), U.moe())],
    "mixture_beside_the_delta_rule": [(U.delta(), U.moe())],
    "mixture_without_groups": [(U.attention(), U.moe(groups=None))],
    "mixture_without_a_shared_expert": [(U.delta(), U.moe(shared=0))],
    "mixture_groups_of_one_expert": [(U.attention(), U.moe(experts=7, top=2, groups=(7, 3)))],
    "mixture_every_group_kept": [(U.attention(), U.moe(experts=8, top=5, groups=(2, 2)))],
    "mixture_one_group_one_expert_chosen": [(U.attention(), U.moe(experts=9, top=1, groups=(3, 1)))],
    "mixture_as_many_chosen_as_kept": [(U.attention(), U.moe(experts=12, top=6, groups=(4, 2), ff=7, shared=3))],
    "mixture_of_forty_in_eight_groups": [(U.attention(), U.moe(experts=40, top=6, groups=(8, 3), ff=8))],
    "mixture_of_sixty_six_without_groups": [(U.delta(), U.moe(experts=66, top=32, groups=None, ff=4))],
}


@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_each_mechanism_alone(name):
    cfg = U.config(MECHANISMS[name])
    W = U.weights(cfg, seed=3)
    t = toks(70, seed=1)
    want = U.oracle_logits(cfg, W, t)
    assert U.rel_err(U.run_whole(cfg, W, t), want) < F32_TOL
    assert U.rel_err(U.run_portions(cfg, W, t, [41, 2, 20]), want) < F32_TOL
    assert U.bf16_close(U.run_whole(cfg, W, t, dtype="bfloat16"), want)


STACK = [(U.delta(), U.moe()), (U.attention(), U.moe(groups=None)), (U.attention(heads=6, kv_heads=3, dim=10, vdim=8, window=7, rot=10, diff=0.7), None),
         (U.delta(heads=2, kv_heads=2, dim=7, vdim=20, conv=5), U.moe(experts=6, top=2, groups=(3, 2), shared=0)), (U.delta(heads=5, kv_heads=1, dim=16, vdim=4, conv=2), None),
         (U.attention(heads=2, kv_heads=1, dim=12, vdim=16, window=33, rot=2, factor=0), U.moe(ff=16))]
LOOP = (1, 4, 2)


def test_every_prefix_of_the_layer_list_matches():
    """Models cut after each layer reproduce the oracle layer by layer."""
    t = toks(45, seed=2)
    full = U.weights(U.config(STACK), seed=5)
    for n in range(1, len(STACK) + 1):
        cfg = U.config(STACK[:n])
        W = {k: v for k, v in full.items() if not k.startswith("l") or int(k[1:k.index(".")]) < n}
        assert U.rel_err(U.run_whole(cfg, W, t), U.oracle_logits(cfg, W, t)) < F32_TOL, n


@pytest.mark.parametrize("loop", [(0, 6, 1), (0, 6, 2), (0, 1, 3), (5, 6, 4), (2, 5, 3)])
def test_loops_of_any_place_and_length(loop):
    """Every pass has its own cache and state, and the embedding joins in front of every pass but the first."""
    cfg = U.config(STACK, loop=loop)
    W = U.weights(cfg, seed=6)
    t = toks(50, seed=3)
    want = U.oracle_logits(cfg, W, t)
    plain = U.oracle_logits(U.config(STACK), W, t)
    assert (U.rel_err(plain, want) > 1e-2) == (loop[2] > 1)
    for cuts in ([50], [20, 2, 3], []):
        assert U.rel_err(U.run_portions(cfg, W, t, cuts), want) < F32_TOL, cuts


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefill_against_token_by_token_decoding(dtype):
    cfg = U.config(STACK, loop=LOOP)
    W = U.weights(cfg, seed=7)
    t = toks(60, seed=3)
    want = U.oracle_logits(cfg, W, t)
    whole = U.run_whole(cfg, W, t, dtype)
    single = U.run_portions(cfg, W, t, [], dtype)
    if dtype == "float32":
        assert U.rel_err(whole, want) < F32_TOL and U.rel_err(single, want) < F32_TOL
    else:
        assert U.bf16_close(whole, want) and U.bf16_close(single, want)
        assert U.bf16_close(whole, single, tol=6e-2)


@pytest.mark.parametrize("sizes", [[2, 2, 2, 3, 2], [5, 1, 17, 2, 40], [64, 2, 63], [1, 70, 2], [33, 33, 33, 33], [23, 2, 24, 25, 47], [129, 2]])
def test_portions_of_several_sizes(sizes):
    """Portions cut anywhere: inside a page (8 tokens), a window (7, 21, 33), the convolution's window (2 to 5), a tile of the
    preparation (16), a group of the recurrence (8) and a key tile (32)."""
    cfg = U.config(STACK, loop=LOOP)
    W = U.weights(cfg, seed=11)
    t = toks(140, seed=4)
    want = U.oracle_logits(cfg, W, t)
    assert U.rel_err(U.run_portions(cfg, W, t, sizes), want) < F32_TOL
    assert U.bf16_close(U.run_portions(cfg, W, t, sizes, "bfloat16"), want)


# bfloat16 with fitting sizes runs on the tensor cores: both maps of the attention, the projections, the bottlenecks' products
TENSOR_CORE_SHAPES = {
    "attention_dim16_values32": [(U.attention(heads=4, kv_heads=4, dim=16, vdim=32, window=100, rot=8), None)],
    "attention_dim24_values48_six_per_group": [(U.attention(heads=6, kv_heads=1, dim=24, vdim=48, window=64, rot=24), None)],
    "attention_dim8_values16_whole_past": [(U.attention(heads=2, kv_heads=1, dim=8, vdim=16, window=0), None)],
    "attention_dim64_values128": [(U.attention(heads=4, kv_heads=2, dim=64, vdim=128, window=130, rot=32), U.moe(ff=64, shared=64)),
                                  (U.attention(heads=4, kv_heads=1, dim=64, vdim=96, window=0, rot=64), None)],
    "attention_dim128_values128": [(U.attention(heads=2, kv_heads=1, dim=128, vdim=128, window=257, rot=64), None)],
    "attention_dim72_values16": [(U.attention(heads=2, kv_heads=2, dim=72, vdim=16, window=33, rot=36), None)],
    "attention_seventy_per_group": [(U.attention(heads=70, kv_heads=1, dim=16, vdim=16, window=300), None)],
    "attention_values_not_a_multiple_of_16": [(U.attention(heads=2, kv_heads=1, dim=16, vdim=24, window=90), None)],
    "delta_dim64_values64": [(U.delta(heads=4, kv_heads=2, dim=64, vdim=64, conv=4, decay_rank=16, gate_rank=32), U.moe(ff=64, shared=64))],
    "delta_dim128_values128": [(U.delta(heads=2, kv_heads=1, dim=128, vdim=128, conv=4, decay_rank=64, gate_rank=24), U.moe(ff=64, shared=64))],
}


@pytest.mark.parametrize("name", sorted(TENSOR_CORE_SHAPES))
def test_tensor_core_shapes(name):
    """Whole prompt, ragged portions (blocks that end inside a key tile or a window) and decoding over a sliced history."""
    cfg = U.config(TENSOR_CORE_SHAPES[name], width=40 if "dim8_" in name else 128)
    W = U.weights(cfg, seed=21)
    t = toks(330, seed=7)
    want = U.oracle_logits(cfg, W, t)
    assert U.rel_err(U.run_portions(cfg, W, t, [100, 3, 150, 64], page_size=16), want) < F32_TOL
    for cuts in ([330], [100, 3, 150, 64], [31, 33, 200, 2, 62], [320]):
        e16 = U.row_errs(U.run_portions(cfg, W, t, cuts, "bfloat16", page_size=16), want)
        assert float(np.quantile(e16, 0.8)) < 3e-2 and float(e16.max()) < 0.4, cuts


def test_attention_over_slices_of_the_history():
    """A single decoding sequence with a long visible history has its keys cut into slices that a second kernel joins -- both maps,
    their difference and its norm.  A layer without a window slices the whole history, one with a long window its window, one with
    a short window not at all, in both compute types and in kernels of both kinds (dim 16 and dim 6)."""
    cfg = U.config([(U.attention(dim=16, vdim=32, window=0, rot=8), None), (U.attention(dim=16, vdim=32, window=300, rot=8), U.moe()), (U.attention(window=0), None),
                    (U.attention(dim=16, vdim=16, window=48, rot=8), None), (U.attention(window=350), None)])
    W = U.weights(cfg, seed=15)
    t = toks(600, seed=6)
    want = U.oracle_logits(cfg, W, t)
    for dtype in ("float32", "bfloat16"):
        e = U.engine(cfg, W, dtype, pool_tokens=640, page_size=64)
        got = U.feed(e, t, [290, 5, 240])  # the portion of 5: one query block over 295 keys -- slices; then 65 decoded tokens
        e.close()
        assert U.rel_err(got, want) < F32_TOL if dtype == "float32" else U.bf16_close(got, want)


RECURRENCE_SHAPES = {  # (dim, vdim): the register shapes of the recurrence, heads in one block of columns and in several
    "dim8_vdim40": (8, 40), "dim48_vdim64": (48, 64), "dim64_vdim96": (64, 96), "dim128_vdim128": (128, 128), "dim20_vdim136": (20, 136),
    "dim130_vdim8": (130, 8), "dim256_vdim24": (256, 24), "dim100_vdim48": (100, 48), "dim32_vdim260": (32, 260), "dim15_vdim131": (15, 131),
    "dim65_vdim17": (65, 17), "dim1_vdim1": (1, 1), "dim33_vdim16": (33, 16),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(RECURRENCE_SHAPES))
def test_state_sizes_of_the_delta_rule(name, dtype):
    """Long spans, spans that continue a state, single tokens, and two sequences of unequal portions in one pass."""
    d, dv = RECURRENCE_SHAPES[name]
    cfg = U.config([(U.delta(heads=4, kv_heads=2, dim=d, vdim=dv, conv=3), None)], width=24)
    W = U.weights(cfg, seed=33)
    a, b = toks(200, seed=11), toks(150, seed=12)
    wa, wb = U.oracle_logits(cfg, W, a), U.oracle_logits(cfg, W, b)
    e = U.engine(cfg, W, dtype, pool_tokens=512, page_size=16, max_batch=2)
    f = U.Feeder(e)
    f.step([("a", a, 130), ("b", b, 20)])
    f.step([("b", b, 1)])
    f.step([("a", a, 69), ("b", b, 8)])
    f.step([("b", b, 1), ("a", a, 1)])
    f.step([("b", b, 120)])
    for key, want in (("a", wa), ("b", wb)):
        got = f.end(key)
        if dtype == "float32":
            assert U.rel_err(got, want) < 5e-5
        else:
            e16 = U.row_errs(got, want)
            assert float(np.quantile(e16, 0.95)) < 3e-2 and float(e16.max()) < 0.3
    e.close()


def test_many_heads_keep_whole_heads_in_a_block():
    """Four prompts of 100 tokens over 40 heads fill the GPU, so a block holds whole heads also in prompts, and the head norm and
    the gate run inside the recurrence."""
    cfg = U.config([(U.delta(heads=40, kv_heads=20, dim=4, vdim=40), None)], width=24)
    W = U.weights(cfg, seed=34)
    seqs = {k: toks(130, seed=50 + k) for k in range(4)}
    e = U.engine(cfg, W, pool_tokens=4 * 144, page_size=16, max_batch=4, max_step_tokens=400)
    f = U.Feeder(e)
    f.step([(k, seqs[k], 100) for k in seqs])
    f.step([(k, seqs[k], 30) for k in seqs])
    for k in seqs:
        assert U.rel_err(f.end(k), U.oracle_logits(cfg, W, seqs[k])) < 5e-5
    e.close()


def test_large_prompt_passes_on_the_persistent_products(monkeypatch):
    """2048 prompt tokens in bfloat16: the experts as a tensor-core product each, the shared expert's gated-unit epilogue, the
    projections on the persistent kernels.  Against the oracle at a few positions, and against the same pass with those kernels off
    (DIS_STACK_PERSIST=0), and with every product on the fp32-FMA kernels (DIS_STACK_TC=0)."""
    cfg = U.config([(U.delta(heads=2, kv_heads=1, dim=16, vdim=16, decay_rank=8, gate_rank=8), U.moe(ff=32, experts=8, top=2, groups=(4, 2), shared=2400)),
                    (U.attention(heads=2, kv_heads=1, dim=16, vdim=32, window=40), U.moe(ff=40, experts=4, top=2, groups=None, shared=64))], width=64, vocab=64)
    W = U.weights(cfg, seed=29)
    seqs = [toks(512, vocab=64, seed=90 + i) for i in range(4)]
    want = np.concatenate([U.oracle_logits(cfg, W, sq[:131])[[7, 130]] for sq in seqs])
    res = []
    for name, flag in ((None, None), ("DIS_STACK_PERSIST", "0"), ("DIS_STACK_TC", "0")):
        if name:
            monkeypatch.setenv(name, flag)
        e = U.engine(cfg, W, "bfloat16", max_batch=4, pool_tokens=4 * 512, page_size=64, max_step_tokens=4 * 512, rows=64)
        P = InferenceParams(max_tokens=1 << 20, temperature=0.0)
        slots = [e.seq_add(sq, P) for sq in seqs]
        for sl in slots:
            e.seq_probe(sl, [7, 130, 300])
        e.step(slots)
        res.append(e.last_logits(e.last_logit_rows()).copy())
        e.close()
        if name:
            monkeypatch.delenv(name)
    assert res[0].shape == (4 * 4, 64)
    first_two = [4 * i + j for i in range(4) for j in (0, 1)]
    for r in res:
        assert U.bf16_close(r[first_two], want)
        assert U.bf16_close(r, res[0], tol=3e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batches_of_unequal_requests_against_each_alone(dtype):
    cfg = U.config(STACK, loop=LOOP)
    W = U.weights(cfg, seed=13)
    seqs = {k: toks(n, seed=20 + i) for i, (k, n) in enumerate([("a", 90), ("b", 33), ("c", 7), ("d", 58)])}
    want = {k: U.oracle_logits(cfg, W, v) for k, v in seqs.items()}
    e = U.engine(cfg, W, dtype, max_batch=4, pool_tokens=512)
    f = U.Feeder(e)
    f.step([("a", seqs["a"], 50), ("b", seqs["b"], 2)])
    f.step([("a", seqs["a"], 1), ("b", seqs["b"], 20), ("c", seqs["c"], 7)])
    f.step([("d", seqs["d"], 30), ("a", seqs["a"], 1), ("b", seqs["b"], 1)])
    while any(f.fed[k] < len(seqs[k]) for k in seqs):
        f.step([(k, seqs[k], min(3 if k == "d" else 1, len(seqs[k]) - f.fed[k])) for k in seqs if f.fed[k] < len(seqs[k])])
    for k in seqs:
        got = f.end(k)
        assert U.rel_err(got, want[k]) < F32_TOL if dtype == "float32" else U.bf16_close(got, want[k]), k
    e.close()


def test_pages_and_slots_are_freed_and_used_again():
    """Two slots and a pool of 12 pages: six sequences pass through them; neither the cached keys nor the recurrent state nor the
    convolution's inputs of the sequence before may reach the next one."""
    cfg = U.config(STACK, loop=LOOP)
    W = U.weights(cfg, seed=17)
    e = U.engine(cfg, W, max_batch=2, pool_tokens=96, page_size=8)
    f = U.Feeder(e)
    lens = [40, 17, 48, 9, 33, 41]
    seqs = [toks(n, seed=40 + i) for i, n in enumerate(lens)]
    live = []
    for i, s in enumerate(seqs):
        if len(live) == 2:
            k = live.pop(0)
            while f.fed[k] < len(seqs[k]):
                f.step([(k, seqs[k], 1)] + [(o, seqs[o], 1) for o in live if f.fed[o] < len(seqs[o])])
            assert U.rel_err(f.end(k), U.oracle_logits(cfg, W, seqs[k])) < F32_TOL, k
        first = [1, 2, len(s) - 5][i % 3]
        f.step([(i, s, first)] + [(o, seqs[o], 1) for o in live if f.fed[o] < len(seqs[o])])
        live.append(i)
    for k in live:
        while f.fed[k] < len(seqs[k]):
            f.step([(k, seqs[k], 1)])
        assert U.rel_err(f.end(k), U.oracle_logits(cfg, W, seqs[k])) < F32_TOL, k
    assert e.status().kv_pages_free == e.status().kv_pages_total
    e.close()


@pytest.mark.parametrize("decode_tail", [0, 40])
def test_far_keys_and_page_borders_with_peaked_weights(decode_tail):
    """A large score scale makes every query put its weight on few keys, wherever in the window they lie: a key that is lost,
    shifted by one or read from the wrong page changes the output by its full size."""
    cfg = U.config([(U.attention(scale=6.0, window=0), None), (U.attention(scale=5.0, window=130), None)])
    W = U.weights(cfg, seed=19, gain=2.0)
    t = toks(300, seed=6)
    want = U.oracle_logits(cfg, W, t)
    e = U.engine(cfg, W, pool_tokens=320, page_size=16)
    got = U.feed(e, t, [300 - decode_tail])
    e.close()
    assert U.rel_err(got, want) < 2e-4


def _planted(n, window, which, heads=2):
    """Hand-made weights for one layer of width n over one-hot inputs (an RMS norm keeps a one-hot row's direction): in map `which` of
    every head the query of token 2 points at the key of token 1; every other query is zero, and so is the other map throughout.  The
    planted pair scores n, every other pair nothing."""
    eye, zero = np.eye(n, dtype=np.float32), np.zeros((n, n), np.float32)
    read = zero.copy()
    read[1, 2] = 1.0
    cfg = U.config([(U.attention(heads=heads, kv_heads=1, dim=n, vdim=n, scale=1.0, window=window, rot=0, diff=0.3), None)], vocab=n, width=n, embed=1.0)
    W = U.weights(cfg, seed=23)
    W["embed"] = eye.copy()
    W["l0.norm1"], W["l0.ls1"] = np.zeros(n, np.float32), np.ones(n, np.float32)
    W["l0.mix.o"] = np.tile(eye * 4.0, (1, heads)).astype(np.float32)
    pair = lambda m: np.concatenate([m, zero] if which == 0 else [zero, m])  # noqa: E731
    W["l0.mix.q"], W["l0.mix.k"], W["l0.mix.v"] = np.tile(pair(read), (heads, 1)), pair(eye), eye.copy()
    return cfg, W


@pytest.mark.parametrize("n,dtype", [(12, "float32"), (16, "bfloat16")])
@pytest.mark.parametrize("which", [0, 1])
def test_a_key_planted_far_back_is_found(which, n, dtype):
    """One key among 260 positions decides the last token's output: at the start of the sequence, on either side of page (16) and
    tile (32, 64) borders, and just before the query."""
    cfg, W = _planted(n, 0, which)
    base = [int(x) for x in np.random.default_rng(1).integers(3, n, 260)]
    base[-1] = 2
    without = U.oracle_logits(cfg, W, base)[-1]
    e = U.engine(cfg, W, dtype, pool_tokens=320, page_size=16)
    for where in (0, 1, 15, 16, 31, 32, 63, 64, 127, 128, 255, 256, 258):
        t = list(base)
        t[where] = 1
        want = U.oracle_logits(cfg, W, t)
        assert np.abs(want[-1] - without).max() > 0.05  # the planted key decides the output
        for tail in (0, 3):  # the query inside a prompt portion, and decoded alone
            assert U.rel_err(U.feed(e, t, [260 - tail]), want) < (1e-4 if dtype == "float32" else 3e-2), (where, tail)
    e.close()


@pytest.mark.parametrize("n,dtype", [(12, "float32"), (16, "bfloat16")])
@pytest.mark.parametrize("which,window", [(0, 100), (1, 64), (0, 37), (1, 1), (0, 2)])
def test_keys_just_inside_and_just_outside_a_window(which, window, n, dtype):
    """The query (last token, position p) sees positions p - window + 1 .. p.  A planted key at the window's first position or the
    one after is seen; one at the position before the window, or two before, is not -- the query's output is then exactly that of the
    sequence without it.  Also when the prompt was cut right at the edge and when the query is decoded alone."""
    cfg, W = _planted(n, window, which)
    e = U.engine(cfg, W, dtype, pool_tokens=448, page_size=16)
    for length in (2 * window + 31, window + 2):
        lo = length - window  # first position the last token sees
        base = [int(x) for x in np.random.default_rng(2).integers(3, n, length)]
        base[-1] = 2
        without = U.oracle_logits(cfg, W, base)
        for where in (lo - 2, lo - 1, lo, lo + 1):
            if where < 0 or where >= length - 1:
                continue
            t = list(base)
            t[where] = 1
            want = U.oracle_logits(cfg, W, t)
            if where >= lo:
                assert np.abs(want[-1] - without[-1]).max() > 0.05
            else:
                assert np.abs(want[-1] - without[-1]).max() == 0.0
            for cuts in ([length], [lo, length - lo], [max(lo - 1, 1), 2, length], [length - 1, 1], [lo + 1, length], [length - 3]):
                got = U.feed(e, t, cuts)
                assert U.rel_err(got, want) < (1e-4 if dtype == "float32" else 3e-2), (length, where, cuts)
    e.close()


def _planted_state(n, taps, delay):
    """Hand-made weights for one delta-rule layer of width n over one-hot inputs: a token 1 writes (`delay` tokens later, through the
    convolution's tap), only token 2 reads there, and next to nothing decays.  Without a token 1 before it, token 2's mixer output
    is zero; with one -- however far back -- it is a vector of fixed size."""
    cfg = U.config([(U.delta(heads=1, kv_heads=1, dim=n, vdim=n, conv=taps), None)], vocab=n, width=n, embed=1.0)
    W = U.weights(cfg, seed=29)
    eye, write, read = np.eye(n, dtype=np.float32), np.zeros((n, n), np.float32), np.zeros((n, n), np.float32)
    write[n - 2, 1], read[n - 2, 2] = 1.0, 1.0
    W["embed"], W["l0.norm1"], W["l0.ls1"] = eye.copy(), np.zeros(n, np.float32), np.ones(n, np.float32)
    W["l0.mix.q"], W["l0.mix.k"], W["l0.mix.v"] = read, write, eye.copy()
    for name, tap in (("q", taps - 1), ("k", taps - 1 - delay), ("v", taps - 1)):
        w = np.zeros((n, taps), np.float32)
        w[:, tap] = 1.0
        W[f"l0.mix.{name}.conv"] = w
    W["l0.mix.dt_bias"] = np.full(n, -16.0, np.float32)
    W["l0.mix.o"] = (eye * 8.0).astype(np.float32)
    return cfg, W


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("taps,delay", [(3, 0), (4, 3), (6, 5)])
def test_state_carried_from_far_back(taps, delay, dtype):
    """Token 1 occurs once among 300 tokens; the last token (2) reads what it left in the state, wherever it stood: at the very
    start, on either side of a border between groups of the recurrence (8) or tiles of the preparation (16), or just before the
    reader -- whole, in portions cut between token 1 and the token that its key reaches, and with the tail decoded."""
    n = 8
    cfg, W = _planted_state(n, taps, delay)
    base = [int(x) for x in np.random.default_rng(5).integers(3, n, 300)]
    base[-1] = 2
    without = U.oracle_logits(cfg, W, base)[-1]
    e = U.engine(cfg, W, dtype, pool_tokens=320, page_size=64)
    for where in (0, 15, 63, 64, 191, 298 - delay):
        t = list(base)
        t[where] = 1
        want = U.oracle_logits(cfg, W, t)
        assert np.abs(want[-1] - without).max() > 0.05  # what token 1 left decides the output
        for cuts in ([300], [3, 250, 2, 40], [where + 1, 64, 2], [where + 1, 1, 1, 1, 1, 1, 1, 200], [296]):
            assert U.rel_err(U.feed(e, t, cuts), want) < (1e-4 if dtype == "float32" else 2e-2), (where, cuts)
    e.close()


def test_the_second_write_at_a_key_replaces_the_first():
    """Two tokens write at one key with step size one (a large logit): the reader gets the second value alone -- what tells the delta
    rule from a plain sum -- also when the two writes come in different passes."""
    n = 8
    cfg, W = _planted_state(n, 2, 0)
    W["l0.mix.k"][n - 2, 3] = 1.0
    W["l0.mix.b"] = np.full((1, n), 8.0, np.float32)
    base = [int(x) for x in np.random.default_rng(6).integers(4, n, 60)]
    base[-1] = 2
    one, both = list(base), list(base)
    both[10], both[40], one[40] = 1, 3, 3
    a, b = U.oracle_logits(cfg, W, one)[-1], U.oracle_logits(cfg, W, both)[-1]
    assert np.abs(a - b).max() < 1e-3 * np.abs(a).max()
    want = U.oracle_logits(cfg, W, both)
    for cuts in ([60], [11, 20, 29], [40]):
        assert U.rel_err(U.run_portions(cfg, W, both, cuts), want) < 1e-4


@pytest.mark.parametrize("experts", [12, 48])
def test_groups_rank_by_their_best_expert_and_weights_leave_the_correction_out(experts):
    """The correction alone decides the choice (router logits are equal): one group has the single best expert, another the best two
    by sum.  Choice scores of the rest are negative, so an excluded expert must count as minus infinity."""
    per = experts // 4
    cfg = U.config([(U.attention(), U.moe(experts=experts, top=3, groups=(4, 1), shared=0))])
    W = U.weights(cfg, seed=51)
    W["l0.mlp.router"] = np.zeros_like(W["l0.mlp.router"])
    c = np.full(experts, -3.0, np.float32)
    c[per], c[2 * per], c[2 * per + 1] = 2.0, 1.75, 1.75
    c[3 * per] = -0.5
    W["l0.mlp.correction"] = models.bf16_round(c)
    t = toks(20, seed=8)
    want = U.oracle_logits(cfg, W, t)
    for cuts in ([20], [9, 2], []):
        assert U.rel_err(U.run_portions(cfg, W, t, cuts), want) < F32_TOL
    W2 = dict(W, **{"l0.mlp.correction": models.bf16_round(np.where(np.arange(experts) // per == 1, c + 5.0, c))})
    assert U.rel_err(U.oracle_logits(cfg, W2, t), want) < 1e-9  # same choice, same weights: the correction is not in them
    W3 = {k: v for k, v in W.items()}
    for e in range(experts):
        if e // per != 1:
            W3[f"l0.mlp.e{e}.down"] = W3[f"l0.mlp.e{e}.down"] * np.float32(64.0)  # nobody outside the best group is asked
    assert U.rel_err(U.run_whole(cfg, W3, t), want) < F32_TOL


def test_first_tokens_of_a_sequence():
    cfg = U.config(STACK, loop=LOOP)
    W = U.weights(cfg, seed=31)
    for n in (1, 2, 3, 5):
        t = toks(n, seed=50 + n)
        assert U.rel_err(U.run_whole(cfg, W, t), U.oracle_logits(cfg, W, t)) < F32_TOL, n
    t = toks(9, seed=60)
    assert U.rel_err(U.run_portions(cfg, W, t, [1, 1, 2, 1, 4]), U.oracle_logits(cfg, W, t)) < F32_TOL


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_keeps_cache_and_state_exact(dtype):
    cfg = U.config([(U.attention(dim=16, vdim=32, window=150, rot=8), U.moe()), (U.delta(), None), (U.attention(window=60), None)], loop=(1, 2, 2))
    W = U.weights(cfg, seed=37)
    t = toks(420, seed=9)
    want = U.oracle_logits(cfg, W, t)
    e = U.engine(cfg, W, dtype, pool_tokens=448, page_size=64)
    got = U.feed(e, t, [20])
    e.close()
    assert U.rel_err(got, want) < 5e-5 if dtype == "float32" else U.bf16_close(got, want)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_positions_in_the_tens_of_thousands_keep_their_angles(dtype):
    """Rotation depends on differences of positions only: a long run of one token followed by a short text gives the logits of the
    text after any other long run of that token (windows and decays have forgotten the difference)."""
    cfg = U.config([(U.attention(dim=16, vdim=32, window=40, rot=16), U.moe()), (U.delta(), None)])
    W = U.weights(cfg, seed=38)
    W["l1.mix.dt_bias"] = np.full_like(W["l1.mix.dt_bias"], 1.0)
    text = toks(30, seed=10)
    outs = []
    for run in (200, 20000):
        t = [7] * run + text
        e = U.engine(cfg, W, dtype, pool_tokens=20096, page_size=64, max_step_tokens=4096, rows=64)
        sl = e.seq_add(t, InferenceParams(max_tokens=1 << 20, temperature=0.0))
        e.seq_probe(sl, list(range(run, run + 30)))
        while True:
            _, _, prod = e.step([sl], 4096)
            if prod[0]:
                break
        outs.append(e.last_logits(e.last_logit_rows())[:30].copy())
        e.close()
    assert U.rel_err(outs[1], outs[0]) < (2e-4 if dtype == "float32" else 5e-2)


ODD = [(U.attention(heads=6, kv_heads=3, dim=10, vdim=14, window=11, rot=6), U.moe(ff=9, experts=5, top=2, groups=(5, 2), shared=1)),
       (U.delta(heads=5, kv_heads=5, dim=7, vdim=3, conv=2, decay_rank=3, gate_rank=2), None),
       (U.attention(heads=1, kv_heads=1, dim=40, vdim=42, window=0, scale=0.9, rot=40, base=9.0, factor=7.5), U.moe(ff=17, groups=None, shared=0)),
       (U.delta(heads=9, kv_heads=3, dim=34, vdim=18, conv=6, decay_rank=40, gate_rank=33), U.moe(experts=34, top=4, groups=(17, 5), ff=5))]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,vocab,eps,embed", [(72, 131, 1e-3, 1.0), (136, 61, 1e-6, 0.25), (50, 33, 1e-5, 6.0), (33, 40, 1e-2, 0.6)])
def test_other_sizes(dtype, width, vocab, eps, embed):
    cfg = U.config(ODD, vocab=vocab, width=width, eps=eps, embed=embed, loop=(1, 3, 2))
    W = U.weights(cfg, seed=41)
    t = toks(75, vocab=vocab, seed=10)
    want = U.oracle_logits(cfg, W, t)
    got = U.run_portions(cfg, W, t, [33, 2, 1, 1, 30, 8], dtype, page_size=16, pool_tokens=128)
    if dtype == "float32":
        assert U.rel_err(got, want) < 5e-5, U.row_errs(got, want)
    else:  # with 34 experts in 17 groups half a percent of noise on the router logits already turns close calls at a fifth of the positions
        e16 = U.row_errs(got, want)
        assert float(np.median(e16)) < 4e-2 and float(e16.max()) < 1.0


def test_model_folder_round_trip(tmp_path):
    """config.json + model.safetensors written by the test, read back through the registry, loaded and run.  The bottlenecks' sizes
    come from the tensors' shapes; a layer without a feed-forward may carry the vectors of one."""
    from tests.test_stack_cpu import write_safetensors
    cfg = U.config(STACK, loop=LOOP)
    W = U.weights(cfg, seed=43)
    for ly in cfg["layers"]:
        ly["mixer"].pop("decay_rank", None)
        ly["mixer"].pop("gate_rank", None)
    extra = {"l2.norm2": np.ones(36, np.float32), "l2.ls2": np.ones(36, np.float32)}
    write_safetensors(tmp_path / "model.safetensors", dict(W, **extra))
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    assert models.read_config(str(tmp_path))[1].name == "Bunosun"
    t = toks(20, seed=12)
    e = models.load_model(str(tmp_path), dtype="float32", max_batch=2, max_tokens=64, page_size=16, max_step_tokens=64, max_logit_rows=68)
    got = U.feed(e, t, [20])
    e.close()
    assert U.rel_err(got, U.oracle_logits(U.config(STACK, loop=LOOP), W, t)) < F32_TOL


def test_greedy_generation_through_the_scheduler():
    """Requests of unequal length through the admission queue and the continuous batcher; greedy tokens equal the oracle's,
    except where the oracle's top two logits are closer than float32 noise."""
    cfg = U.config(STACK, vocab=40, loop=LOOP)
    W = U.weights(cfg, seed=43)
    e = U.engine(cfg, W, max_batch=3, pool_tokens=256, page_size=8, max_step_tokens=64)
    cb = ContinuousBatcher(e, max_active=3)
    cb.set_prefill_budget(16)  # prompts are read in portions beside the running sequences
    prompts = [toks(n, vocab=40, seed=70 + n) for n in (5, 37, 12, 1, 26)]
    new = [9, 6, 12, 7, 5]
    for i, p in enumerate(prompts):
        cb.submit(i, p, InferenceParams(new[i], 0.0))
    res = cb.run_until_idle()
    for i, p in enumerate(prompts):
        seq = list(p)
        got = res[i]["tokens"]
        assert len(got) == new[i]
        for j in range(new[i]):
            lg = U.oracle_logits(cfg, W, seq)[-1]
            top2 = np.sort(lg)[-2:]
            if int(np.argmax(lg)) != got[j]:
                assert top2[1] - top2[0] < 1e-4, (i, j)
            seq.append(got[j])
    cb.close()
    e.close()


def test_parallel_layers_with_two_norms_take_dense_units_too():
    """The frame is not tied to the mixture: the same layers with a dense SiLU unit, in both compute types, whole and decoded."""
    cfg = U.config([(U.attention(), U.moe()), (U.delta(), U.moe())], width=48)
    spec = models.bunosun_spec(cfg)
    for L in spec.layers:
        L.mlp, L.ff, L.route, L.experts, L.top, L.shared_ff = "dense", 56, "softmax_top", 0, 0, 0
    rng = np.random.default_rng(5)
    W = {k: v for k, v in U.weights(cfg, seed=3).items() if ".mlp." not in k}
    for i in range(2):
        for nm, sh in (("gate", (56, 48)), ("up", (56, 48)), ("down", (48, 56))):
            W[f"l{i}.mlp.{nm}"] = models.bf16_round(rng.normal(0, sh[1] ** -0.5, sh).astype(np.float32))
    from distributed_inference_server_b200 import Engine, WorkerConfig
    from tests import bunosun_oracle as BO
    P = {k: np.asarray(v, np.float64) for k, v in W.items()}
    t = toks(90, seed=4)
    x = P["embed"][t] * cfg["embedding"]["scale"]
    eps = cfg["norm"]["eps"]
    for i, ly in enumerate(cfg["layers"]):
        p = f"l{i}."
        mix = BO.attention if ly["type"] == "attention" else BO.channel_delta
        x = x + (mix(ly["mixer"], P, p + "mix.", BO.rms_norm_around_one(x, P[p + "norm1"], eps), eps) * P[p + "ls1"] +
                 BO.gated_unit(P, p + "mlp.", BO.rms_norm_around_one(x, P[p + "norm2"], eps)) * P[p + "ls2"])
    want = BO.rms_norm_around_one(x, P["final.norm"], eps) @ P["head"].T
    for dtype in ("float32", "bfloat16"):
        e = Engine(WorkerConfig(None, max_batch=2, max_step_tokens=128, page_size=8, kv_pages=16, stack=spec, context_size=128, compute_dtype=dtype, max_logit_rows=130))
        for name, a in W.items():
            e.load_named(name, a)
        e.finalize()
        for cuts in ([90], [70, 2]):
            got = U.feed(e, t, cuts)
            assert U.rel_err(got, want) < (F32_TOL if dtype == "float32" else 4e-2), cuts
        e.close()


def test_engine_refuses_what_it_cannot_run():
    from distributed_inference_server_b200 import Engine, WorkerConfig
    from distributed_inference_server_b200 import binding as B

    def make(spec):
        Engine(WorkerConfig(None, max_batch=2, kv_pages=4, page_size=8, stack=spec, context_size=32, compute_dtype="float32"))
    spec = models.bunosun_spec(U.config([(U.delta(), None)]))
    spec.two_norms = spec.layer_scale = spec.loop_embed = False
    with pytest.raises(Exception, match="two norms"):
        make(spec)
    spec = models.bunosun_spec(U.config([(U.attention(), None)]))
    spec.layers[0].attn_flags |= B.ATTN_SINK
    with pytest.raises(Exception, match="plain softmax"):
        make(spec)
    with pytest.raises(Exception, match="dim up to 256"):
        make(models.bunosun_spec(U.config([(U.delta(dim=260), None)])))
    spec = models.bunosun_spec(U.config([(U.attention(), None)], loop=(0, 1, 2)))
    spec.loop_plain = False
    with pytest.raises(Exception, match="loop"):
        make(spec)


def _random_model(rng):
    """A made-up configuration: any order of the two mixers, any window, sizes of heads, states, bottlenecks and experts, with and
    without feed-forwards, loops, groups and shared experts."""
    width, vocab = int(rng.choice([48, 64, 96, 128, 200, 50])), int(rng.integers(40, 300))
    layers = []
    for _ in range(int(rng.integers(2, 6))):
        g = int(rng.choice([1, 2, 3]))
        if rng.random() < 0.5:
            d = int(rng.choice([6, 8, 16, 24, 64]))
            mx = U.attention(heads=g * int(rng.choice([1, 2, 4])), kv_heads=g, dim=d, vdim=int(rng.choice([5, 16, 32, 64, 128])), window=int(rng.choice([0, 1, 7, 33, 64, 100])),
                             rot=int(rng.choice([0, 2, d // 2, d])) // 2 * 2, base=float(rng.choice([10.0, 1e4, 1e6])), factor=float(rng.choice([0, 1.0, 8.0])), diff=float(rng.choice([0.2, 0.8])))
        else:
            mx = U.delta(heads=g * int(rng.choice([1, 2])), kv_heads=g, dim=int(rng.choice([4, 8, 16, 40, 64, 128])), vdim=int(rng.choice([4, 8, 24, 64, 144])),
                         conv=int(rng.choice([1, 2, 3, 4, 5])), decay_rank=int(rng.choice([3, 8, 24])), gate_rank=int(rng.choice([2, 16, 40])))
        gr = int(rng.choice([1, 2, 4]))
        experts = gr * int(rng.choice([2, 3, 10]))
        keep = int(rng.integers(1, gr + 1))
        ml = U.moe(ff=int(rng.choice([8, 24, 33])), experts=experts, top=min(int(rng.choice([1, 2, 4])), keep * (experts // gr)), groups=(gr, keep) if rng.random() < 0.7 else None,
                   shared=int(rng.choice([0, 8, 21])))
        layers.append((mx, None if rng.random() < 0.25 else ml))
    a = int(rng.integers(0, len(layers)))
    loop = (a, int(rng.integers(a + 1, len(layers) + 1)), int(rng.integers(1, 4))) if rng.random() < 0.6 else None
    return U.config(layers, vocab=vocab, width=width, eps=float(rng.choice([1e-5, 1e-3])), embed=float(rng.choice([1.0, 0.5, 3.0])), loop=loop)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(6))
def test_random_configurations_and_schedules(seed, dtype):
    """Up to four live requests, random portions beside single tokens, requests left out of a step, a pool that makes pages and
    slots go round: every position's logits against the oracle."""
    rng = np.random.default_rng(7000 + seed)
    cfg = _random_model(rng)
    W = U.weights(cfg, seed=seed)
    seqs = {k: toks(int(rng.choice([1, 2, 5, 23, 64, 65, 130, 200])), vocab=cfg["vocab"], seed=seed * 10 + k) for k in range(int(rng.integers(3, 7)))}
    want = {k: U.oracle_logits(cfg, W, v) for k, v in seqs.items()}
    page = int(rng.choice([8, 16, 64]))
    pool = sum((n + page - 1) // page * page for n in sorted((len(v) for v in seqs.values()), reverse=True)[:4]) + page
    e = U.engine(cfg, W, dtype, max_batch=4, pool_tokens=pool, page_size=page, max_step_tokens=pool)
    f = U.Feeder(e)
    waiting, live, got = list(seqs), [], {}
    while waiting or live:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
        step = []
        for k in live:
            rem = len(seqs[k]) - f.fed.get(k, 0)
            if rng.random() < 0.15 and len(live) > 1 and f.fed.get(k, 0) > 0:
                continue  # left out of this step
            r = rng.random()
            step.append((k, seqs[k], 1 if r < 0.4 else int(rng.integers(1, rem + 1)) if r < 0.8 else rem))
        if not step:
            continue
        f.step(step)
        for k, _, _ in step:
            if f.fed[k] == len(seqs[k]):
                got[k] = f.end(k)
                live.remove(k)
    assert e.status().kv_pages_free == e.status().kv_pages_total
    e.close()
    for k in seqs:
        if dtype == "float32":
            assert U.rel_err(got[k], want[k]) < 1e-4, (seed, k)
        else:
            # a close call of a router goes the other way now and then, and the states carry the difference on for a while
            e16 = U.row_errs(got[k], want[k])
            assert float(np.median(e16)) < 6e-2 and float(e16.max()) < 1.2, (seed, k)
