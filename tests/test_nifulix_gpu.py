"""Nifulix on the GPU against the float64 oracle (tests/nifulix_oracle.py): small made-up configurations with random or hand-made
weights.  Covered: each mechanism alone, the model layer by layer, prefill against token-by-token decoding, portions down to two
tokens, unequal batches, reuse of pages and slots, keys far back / at page borders / just inside and just outside a window and
among the kept first positions, state carried from far back, value mixing, the first tokens, long decoding, long spans through the
segment path of the recurrence, other sizes, the tensor-core paths of prompt passes, a model folder, and greedy generation
through the scheduler."""
import json

import numpy as np
import pytest

from distributed_inference_server_b200 import ContinuousBatcher, InferenceParams, models
from tests import _nifulix_util as U

pytestmark = pytest.mark.gpu
F32_TOL = 2e-5


def toks(n, vocab=50, seed=0):
    return [int(x) for x in np.random.default_rng(seed).integers(0, vocab, n)]


MECHANISMS = {
    "attention_whole_past": [(U.attention(window=0), None)],
    "attention_window_of_five_keep_none": [(U.attention(window=5, keep=0), None)],
    "attention_window_of_one_keep_one": [(U.attention(window=1, keep=1), None)],
    "attention_window_of_seven_keep_forty": [(U.attention(window=7, keep=40), None)],
    "attention_no_cap": [(U.attention(softcap=0), None)],
    "attention_tight_cap": [(U.attention(softcap=0.3, scale=2.0), None)],
    "attention_one_kv_head_wider_values": [(U.attention(heads=3, kv_heads=1, dim=6, vdim=10, window=17), None)],
    "attention_as_many_kv_heads": [(U.attention(heads=2, kv_heads=2, dim=10, vdim=4, window=64), None)],
    "attention_mixed_values": [(U.attention(), None), (U.attention(heads=6, dim=4, vdim=8), None)],
    "attention_first_layer_does_not_mix": [(U.attention(v_mix=False, vdim=6), None), (U.attention(), None), (U.retention(), None), (U.attention(window=9), None)],
    "retention_alone": [(U.retention(), None)],
    "retention_every_coordinate_rotated": [(U.retention(heads=3, dim=10, vdim=4, rot=10, base=77.0), None)],
    "retention_nothing_rotated": [(U.retention(heads=1, dim=6, vdim=14, rot=0), None)],
    "retention_fast_and_no_decay": [(U.retention(heads=4, decay=[0.0, 0.3, 0.9, 1.0]), None)],
    "latent_alone": [(U.latent(), None)],
    "latent_whole_past": [(U.latent(window=0), None)],
    "latent_window_of_one": [(U.latent(window=1), None)],
    "latent_one_head_rank_one_query": [(U.latent(heads=1, dim=3, rot_dim=6, vdim=5, kv_rank=7, q_rank=1), None)],
    "latent_queries_without_a_latent": [(U.latent(q_rank=0), None)],
    "dense_unit_beside_attention": [(U.attention(), U.dense(ff=36))],
    "dense_unit_beside_retention": [(U.retention(), U.dense(ff=7))],
    "dense_unit_beside_latent": [(U.latent(), U.dense(ff=41))],
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


STACK = [(U.attention(), U.dense()), (U.retention(), U.dense(ff=18)), (U.latent(), None), (U.attention(heads=6, kv_heads=2, dim=10, vdim=8, window=7, keep=5, softcap=3.0), U.dense()),
         (U.latent(heads=5, dim=4, rot_dim=6, vdim=7, kv_rank=12, q_rank=9, window=40), U.dense(ff=30)), (U.retention(heads=5, dim=6, vdim=9, rot=2), None),
         (U.attention(heads=2, kv_heads=1, dim=12, vdim=16, window=33, keep=9), U.dense(ff=16))]


def test_every_prefix_of_the_layer_list_matches():
    """Models cut after each layer reproduce the oracle layer by layer."""
    t = toks(45, seed=2)
    full = U.weights(U.config(STACK), seed=5)
    for n in range(1, len(STACK) + 1):
        cfg = U.config(STACK[:n])
        W = {k: v for k, v in full.items() if not k.startswith("l") or int(k[1:k.index(".")]) < n}
        assert U.rel_err(U.run_whole(cfg, W, t), U.oracle_logits(cfg, W, t)) < F32_TOL, n


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefill_against_token_by_token_decoding(dtype):
    cfg = U.config(STACK)
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
    """Portions cut anywhere: inside a page (8 tokens), a window (7, 19, 24, 33, 40), the kept first positions (3, 5, 9), a segment
    of the recurrence (64) and a key tile (32)."""
    cfg = U.config(STACK)
    W = U.weights(cfg, seed=11)
    t = toks(140, seed=4)
    want = U.oracle_logits(cfg, W, t)
    assert U.rel_err(U.run_portions(cfg, W, t, sizes), want) < F32_TOL
    assert U.bf16_close(U.run_portions(cfg, W, t, sizes, "bfloat16"), want)


# bfloat16 with fitting sizes runs on the tensor cores: attention and latent attention, the parallel layer's fused products
TENSOR_CORE_SHAPES = {
    "attention_dim16_window100_keep70": [(U.attention(heads=4, kv_heads=4, dim=16, window=100, keep=70), None)],
    "attention_dim32_values16_six_per_group": [(U.attention(heads=6, kv_heads=1, dim=32, vdim=16, window=64, keep=1), None)],
    "attention_dim80_whole_past_no_cap": [(U.attention(heads=2, kv_heads=1, dim=80, window=0, softcap=0), None)],
    "attention_dim128_two_windows_mixed": [(U.attention(heads=8, kv_heads=2, dim=128, window=257, keep=4), U.dense(64)), (U.attention(heads=8, kv_heads=2, dim=128, window=33, keep=66), U.dense(64))],
    "attention_seventy_per_group": [(U.attention(heads=70, kv_heads=1, dim=16, window=300, keep=2), None)],
    "latent_rank32": [(U.latent(heads=4, dim=16, rot_dim=16, vdim=16, kv_rank=32, q_rank=24, window=70), U.dense(64))],
    "latent_twenty_heads": [(U.latent(heads=20, dim=8, rot_dim=8, vdim=8, kv_rank=24, q_rank=16, window=100), None)],
    "latent_whole_past": [(U.latent(heads=3, dim=24, rot_dim=16, vdim=40, kv_rank=48, q_rank=40, window=0), None)],
    "latent_wide_heads": [(U.latent(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=64, q_rank=72, window=130), U.dense(128))],
    "latent_values_not_a_multiple_of_16": [(U.latent(heads=2, dim=16, rot_dim=8, vdim=24, kv_rank=40, q_rank=16, window=90), None)],
    "latent_windows_of_two_sizes": [(U.latent(heads=4, dim=16, rot_dim=16, vdim=16, kv_rank=32, q_rank=24, window=31), None), (U.latent(heads=2, dim=16, rot_dim=16, vdim=32, kv_rank=32, q_rank=24, window=200), None)],
    "retention_dim64": [(U.retention(heads=2, dim=64, vdim=64, rot=32), U.dense(64))],
}


@pytest.mark.parametrize("name", sorted(TENSOR_CORE_SHAPES))
def test_tensor_core_shapes(name):
    """Whole prompt, ragged portions (blocks that end inside a key tile or a window) and decoding over a sliced history."""
    cfg = U.config(TENSOR_CORE_SHAPES[name], width=40)
    W = U.weights(cfg, seed=21)
    t = toks(330, seed=7)
    want = U.oracle_logits(cfg, W, t)
    assert U.rel_err(U.run_portions(cfg, W, t, [100, 3, 150, 64], page_size=16), want) < F32_TOL
    for cuts in ([330], [100, 3, 150, 64], [31, 33, 200, 2, 62], [320]):
        e16 = U.row_errs(U.run_portions(cfg, W, t, cuts, "bfloat16", page_size=16), want)
        assert float(np.quantile(e16, 0.8)) < 3e-2 and float(e16.max()) < 0.3, cuts


LATENT_ROUTES = {  # how prompt portions of latent layers run in bfloat16: per-head keys and values; products over the latents; both in one pass
    "per_head": {}, "products": {"DIS_STACK_LATENT_FLASH": "0"}, "rows_for_one_span": {"DIS_STACK_LATENT_ROWS": "152"}, "rows_for_short_spans_only": {"DIS_STACK_LATENT_ROWS": "104"},
    "fp32_products": {"DIS_STACK_TC": "0"},
}


@pytest.mark.parametrize("route", sorted(LATENT_ROUTES))
def test_prompt_portions_of_latent_layers(route, monkeypatch):
    """Four sequences' portions beside a decoded token in one pass, with histories: all through per-head keys and values in one
    group or a group per span, through the products over the latents, or span by span either way (a span with more keys than rows)."""
    for k, v in LATENT_ROUTES[route].items():
        monkeypatch.setenv(k, v)
    cfg = U.config([(U.latent(heads=4, dim=16, rot_dim=16, vdim=16, kv_rank=32, q_rank=24, window=0), U.dense(24)), (U.latent(heads=3, dim=24, rot_dim=8, vdim=32, kv_rank=40, q_rank=16, window=70), None),
                    (U.latent(heads=2, dim=8, rot_dim=8, vdim=16, kv_rank=24, q_rank=0, window=50), U.dense(24))], width=40)
    W = U.weights(cfg, seed=22)
    seqs = {k: toks(n, seed=60 + k) for k, n in enumerate((150, 140, 100, 90, 60))}
    want = {k: U.oracle_logits(cfg, W, v) for k, v in seqs.items()}
    e = U.engine(cfg, W, "bfloat16", max_batch=5, pool_tokens=640, page_size=16, max_step_tokens=300)
    f = U.Feeder(e)
    f.step([(0, seqs[0], 100), (1, seqs[1], 33), (4, seqs[4], 31)])
    f.step([(1, seqs[1], 70), (0, seqs[0], 1), (2, seqs[2], 64), (4, seqs[4], 1), (3, seqs[3], 40)])
    f.step([(0, seqs[0], 49), (4, seqs[4], 1), (1, seqs[1], 37), (2, seqs[2], 36), (3, seqs[3], 50)])
    f.step([(4, seqs[4], 27)])
    for k in seqs:
        e16 = U.row_errs(f.end(k), want[k])
        assert float(e16.max()) < 3e-2, (route, k, int(e16.argmax()))
    e.close()


def test_attention_over_slices_of_the_history():
    """A single decoding sequence with a long visible history has its keys cut into slices that a second kernel merges.  A layer
    without a window slices the whole history, one with a long window its window and the kept positions, one with a short window
    not at all; latent layers likewise -- all in one model, in prompts and in decoding, in both compute types."""
    cfg = U.config([(U.attention(dim=16, window=0), None), (U.attention(dim=16, window=300, keep=50), U.dense()), (U.attention(dim=16, window=48), None),
                    (U.latent(heads=4, dim=16, rot_dim=16, vdim=16, kv_rank=32, window=0), None), (U.latent(heads=4, dim=16, rot_dim=16, vdim=16, kv_rank=32, window=350), None)])
    W = U.weights(cfg, seed=15)
    t = toks(600, seed=6)
    want = U.oracle_logits(cfg, W, t)
    for dtype in ("float32", "bfloat16"):
        e = U.engine(cfg, W, dtype, pool_tokens=640, page_size=64)
        got = U.feed(e, t, [290, 5, 240])  # the portion of 5: one query block over 295 keys -- slices; then 65 decoded tokens
        e.close()
        assert U.rel_err(got, want) < F32_TOL if dtype == "float32" else U.bf16_close(got, want)


RECURRENCE_SHAPES = {  # (dim, vdim): the register shapes of the recurrence kernel, value columns in blocks, its shared-memory form
    "dim8_vdim40": (8, 40), "dim48_vdim64": (48, 64), "dim64_vdim96": (64, 96), "dim128_vdim128": (128, 128), "dim20_vdim136": (20, 136),
    "dim130_vdim8": (130, 8), "dim128_vdim64": (128, 64), "dim100_vdim48": (100, 48), "dim32_vdim260": (32, 260), "dim16_vdim131": (16, 131),
    "dim64_vdim16": (64, 16), "dim96_vdim112": (96, 112),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(RECURRENCE_SHAPES))
def test_long_spans_through_the_segments_of_the_recurrence(name, dtype):
    """Spans longer than 64 tokens can run as segments side by side joined by a carry; spans of 64 and fewer run in one piece; both
    must agree with the token-by-token oracle, also when a span continues a state (the second portion) and in a batch of two."""
    d, dv = RECURRENCE_SHAPES[name]
    cfg = U.config([(U.retention(heads=2, dim=d, vdim=dv, rot=d // 4 * 2, decay=[0.97, 0.9995]), None)], width=24)
    W = U.weights(cfg, seed=33)
    a, b = toks(200, seed=11), toks(150, seed=12)
    wa, wb = U.oracle_logits(cfg, W, a), U.oracle_logits(cfg, W, b)
    e = U.engine(cfg, W, dtype, pool_tokens=512, page_size=16, max_batch=2)
    f = U.Feeder(e)
    f.step([("a", a, 130), ("b", b, 20)])
    f.step([("a", a, 70), ("b", b, 129)])
    f.step([("b", b, 1)])
    for key, want in (("a", wa), ("b", wb)):
        got = f.end(key)
        if dtype == "float32":
            assert U.rel_err(got, want) < 5e-5
        else:
            assert U.row_errs(got, want).max() < 3e-2
    e.close()


@pytest.mark.parametrize("force", ["1", "2"])
def test_many_heads_and_sequences_walk_long_spans_whole(monkeypatch, force):
    """Four prompts of 100 tokens over 40 heads fill the GPU span by span, so the pass walks each span in one piece although
    it is longer than a segment; DIS_STACK_LIGHT_SEGMENTS=2 cuts it all the same."""
    monkeypatch.setenv("DIS_STACK_LIGHT_SEGMENTS", force)
    cfg = U.config([(U.retention(heads=40, dim=4, vdim=4, rot=4, decay=[1 - 0.5 / (h + 1) for h in range(40)]), None)], width=24)
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
    """2048 prompt tokens in bfloat16 through parallel layers wide enough for the persistent tensor-core products, whose gated-unit
    epilogue writes into the columns behind the mixer's.  Against the oracle at a few positions, and against the same pass with
    those kernels off (DIS_STACK_PERSIST=0), and with every product on the fp32-FMA kernels (DIS_STACK_TC=0)."""
    cfg = U.config([(U.retention(heads=2, dim=16, vdim=16, rot=8), U.dense(ff=2400)), (U.attention(heads=2, kv_heads=1, dim=16, window=40), U.dense(ff=2400)),
                    (U.latent(heads=4, dim=16, rot_dim=16, vdim=16, kv_rank=32, q_rank=16, window=60), U.dense(ff=2400))], width=64, vocab=64)
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
    cfg = U.config(STACK)
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
    """Two slots and a pool of 12 pages: six sequences pass through them; neither the cached keys and latents nor the recurrent
    state of the sequence before may reach the next one."""
    cfg = U.config(STACK)
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


PEAKED = {"attention": [(U.attention(scale=6.0, window=0, softcap=200.0), None), (U.attention(scale=5.0, window=130, keep=20, softcap=150.0), None)],
          "latent": [(U.latent(scale=1.5, window=130), None), (U.latent(scale=1.5, window=0), None)]}


@pytest.mark.parametrize("decode_tail", [0, 40])
@pytest.mark.parametrize("kind", sorted(PEAKED))
def test_far_keys_and_page_borders_with_peaked_weights(kind, decode_tail):
    """A large score scale makes every query put its weight on few keys, wherever in the window they lie: a key that is lost,
    shifted by one or read from the wrong page changes the output by its full size."""
    cfg = U.config(PEAKED[kind])
    W = U.weights(cfg, seed=19, gain=2.0)
    t = toks(300, seed=6)
    want = U.oracle_logits(cfg, W, t)
    e = U.engine(cfg, W, pool_tokens=320, page_size=16)
    got = U.feed(e, t, [300 - decode_tail])
    e.close()
    assert U.rel_err(got, want) < 2e-4


def _planted(kind, n, window, keep=0, heads=1, scale=1.0):
    """Hand-made weights for one layer of width n over one-hot inputs (an RMS norm keeps a one-hot row's direction): the query of
    token 2 points, in every head, at the key of token 1; every other token's query is zero.  The planted pair scores n * scale
    (less the distance term), every other pair nothing."""
    eye, zero = np.eye(n, dtype=np.float32), np.zeros((n, n), np.float32)
    read = zero.copy()
    read[1, 2] = 1.0
    if kind == "attention":
        cfg = U.config([(U.attention(heads=heads, kv_heads=1, dim=n, scale=scale, window=window, keep=keep, softcap=0), None)], vocab=n, width=n, mult=1.0)
    else:
        cfg = U.config([(U.latent(heads=heads, dim=n, rot_dim=n, vdim=n, kv_rank=n, q_rank=n, scale=scale, window=window), None)], vocab=n, width=n, mult=1.0)
    W = U.weights(cfg, seed=23)
    W["embed"] = eye.copy()
    W["l0.norm1"] = np.zeros(n, np.float32)
    W["l0.mix.o"] = np.tile(eye * 64.0, (1, heads)).astype(np.float32)
    if kind == "attention":
        W["l0.mix.q"], W["l0.mix.k"], W["l0.mix.v"] = np.tile(read, (heads, 1)), eye.copy(), eye.copy()
        W["l0.mix.g"] = np.zeros((heads * n, n), np.float32)  # every gate one half
    else:
        W["l0.mix.dq"] = read.copy()
        W["l0.mix.dq.norm"] = W["l0.mix.dkv.norm"] = np.ones(n, np.float32)
        W["l0.mix.uq"] = np.tile(np.concatenate([eye, zero]), (heads, 1))  # [unrotated, rotated] per head
        W["l0.mix.dkv"] = np.concatenate([eye, zero])
        W["l0.mix.uk"] = W["l0.mix.uv"] = np.tile(eye, (heads, 1))
    return cfg, W


@pytest.mark.parametrize("kind,n,dtype", [("attention", 12, "float32"), ("attention", 16, "bfloat16"), ("latent", 12, "float32"), ("latent", 16, "bfloat16")])
def test_a_key_planted_far_back_is_found(kind, n, dtype):
    """One key among 260 positions decides the last token's output: at the start of the sequence, on either side of page (16) and
    tile (32, 64) borders, and just before the query."""
    cfg, W = _planted(kind, n, window=0)
    base = [int(x) for x in np.random.default_rng(1).integers(3, n, 260)]
    base[-1] = 2
    without = U.oracle_logits(cfg, W, base)[-1]
    e = U.engine(cfg, W, dtype, pool_tokens=320, page_size=16)
    for where in (0, 1, 15, 16, 31, 32, 63, 64, 65, 127, 128, 200, 255, 256, 257, 258):
        t = list(base)
        t[where] = 1
        want = U.oracle_logits(cfg, W, t)
        assert np.abs(want[-1] - without).max() > 0.05  # the planted key decides the output
        for tail in (0, 3):  # the query inside a prompt portion, and decoded alone
            assert U.rel_err(U.feed(e, t, [260 - tail]), want) < (1e-4 if dtype == "float32" else 2e-2), (where, tail)
    e.close()


@pytest.mark.parametrize("kind,n,dtype", [("attention", 12, "float32"), ("attention", 16, "bfloat16"), ("latent", 12, "float32"), ("latent", 16, "bfloat16")])
@pytest.mark.parametrize("window", [100, 64, 37])
def test_keys_just_inside_and_just_outside_a_window(kind, n, dtype, window):
    """The query (last token, position p) sees positions p - window + 1 .. p and the kept first ones.  A planted key at the window's
    first position or the one after is seen; one at the position before the window, or two before, is not -- the query's output is
    then exactly that of the sequence without it.  Likewise the last kept position is seen from afar and the next one is not.  Also
    when the prompt was cut right at the edge and when the query is decoded alone."""
    keep = 5 if kind == "attention" else 0
    cfg, W = _planted(kind, n, window, keep=keep)
    e = U.engine(cfg, W, dtype, pool_tokens=448, page_size=16)
    for length in (2 * window + 31, 3 * window + 1, window + 2):
        lo = length - window  # first position the last token sees
        base = [int(x) for x in np.random.default_rng(2).integers(3, n, length)]
        base[-1] = 2
        without = U.oracle_logits(cfg, W, base)
        for where in sorted({lo - 2, lo - 1, lo, lo + 1, 0, keep - 1, keep, keep + 1}):
            if where < 0 or where >= length - 1:
                continue
            t = list(base)
            t[where] = 1
            want = U.oracle_logits(cfg, W, t)
            if where >= lo or where < keep:
                assert np.abs(want[-1] - without[-1]).max() > 0.05
            else:
                assert np.abs(want[-1] - without[-1]).max() == 0.0
            for cuts in ([length], [lo, length - lo], [max(lo - 1, 1), 2, length], [length - 1, 1], [lo + 1, length], [length - 3]):
                got = U.feed(e, t, cuts)
                assert U.rel_err(got, want) < (1e-4 if dtype == "float32" else 2e-2), (length, where, cuts)
    e.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_distance_term_and_the_cap(dtype):
    """Token 1 stands at several distances from the query, its score capped or not: what decides is how far the slope has lowered
    it against the keys beside the query.  Two heads with slopes 2^-4 and 2^-8; the cap comes before the distance term."""
    n = 16
    outs = []
    for cap in (0.0, 6.0):
        cfg, W = _planted("attention", n, window=0, heads=2)
        cfg["layers"][0]["mixer"]["softcap"] = cap
        W["l0.mix.o"][:, n:] = 32.0 * np.roll(np.eye(n, dtype=np.float32), 1, axis=0)  # the heads' outputs land in different places
        e = U.engine(cfg, W, dtype, pool_tokens=320, page_size=16)
        for dist in (1, 40, 90, 230):
            t = [int(x) for x in np.random.default_rng(4).integers(3, n, 250)]
            t[249 - dist], t[-1] = 1, 2
            want = U.oracle_logits(cfg, W, t)
            outs.append(want[-1])
            for cuts in ([250], [200, 49]):
                assert U.rel_err(U.feed(e, t, cuts), want) < (1e-4 if dtype == "float32" else 2e-2), (cap, dist, cuts)
        e.close()
    assert all(np.abs(outs[4 + i] - outs[4 + j]).max() > 0.3 for i in range(4) for j in range(i))  # capped: every distance tells
    assert np.abs(outs[0] - outs[3]).max() > 0.3 and all(np.abs(outs[i] - outs[4 + i]).max() > 0.3 for i in (1, 2, 3))


def test_values_come_from_the_first_mixing_layer_of_the_same_token():
    """With a weight of one a later layer's values are wholly the first mixing layer's -- not the first attention layer's, and not
    its own, whatever its own projection says; the mixed values are what later tokens find in the cache."""
    cfg = U.config([(U.attention(v_mix=False), None), (U.retention(), None), (U.attention(), None), (U.attention(), U.dense()), (U.attention(), None)])
    W = U.weights(cfg, seed=47)
    W["l3.mix.vmix"] = np.float32(1.0)
    t = toks(60, seed=9)
    want = U.oracle_logits(cfg, W, t)
    for scale in (1.0, 64.0):
        W2 = dict(W, **{"l3.mix.v": W["l3.mix.v"] * np.float32(scale)})
        for cuts in ([60], [20, 2, 30], []):
            assert U.rel_err(U.run_portions(cfg, W2, t, cuts), want) < F32_TOL
    W3 = dict(W, **{"l2.mix.v": W["l2.mix.v"] * np.float32(2.0)})
    assert U.rel_err(U.oracle_logits(cfg, W3, t), want) > 1e-3


def _planted_state(n):
    """Hand-made weights for one retention layer of width n over one-hot inputs: only token 1 writes (a key along an unrotated
    coordinate), only token 2 reads there, and next to nothing decays.  Without a token 1 before it, token 2's mixer output is zero;
    with one -- however far back -- it is a vector of fixed size."""
    cfg = U.config([(U.retention(heads=1, dim=n, vdim=n, rot=n // 2, decay=[0.9999]), None)], vocab=n, width=n, mult=1.0)
    W = U.weights(cfg, seed=29)
    eye, write, read = np.eye(n, dtype=np.float32), np.zeros((n, n), np.float32), np.zeros((n, n), np.float32)
    write[n - 2, 1], read[n - 2, 2] = 1.0, 1.0
    W["embed"], W["l0.norm1"] = eye.copy(), np.zeros(n, np.float32)
    W["l0.mix.q"], W["l0.mix.k"], W["l0.mix.v"] = read, write, eye.copy()
    W["l0.mix.g"], W["l0.mix.o"] = np.ones((n, n), np.float32), (eye * 64.0).astype(np.float32)
    return cfg, W


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_state_carried_from_far_back(dtype):
    """Token 1 occurs once among 300 tokens; the last token (2) reads what it left in the state, wherever it stood: at the very
    start, on either side of a border between segments of the recurrence, or just before the reader -- whole, in ragged
    portions, and with the tail decoded through the slot's state."""
    n = 8
    cfg, W = _planted_state(n)
    base = [int(x) for x in np.random.default_rng(5).integers(3, n, 300)]
    base[-1] = 2
    without = U.oracle_logits(cfg, W, base)[-1]
    e = U.engine(cfg, W, dtype, pool_tokens=320, page_size=64)
    for where in (0, 63, 64, 65, 191, 298):
        t = list(base)
        t[where] = 1
        want = U.oracle_logits(cfg, W, t)
        assert np.abs(want[-1] - without).max() > 0.05  # what token 1 left decides the output
        for cuts in ([300], [3, 250, 2, 40], [where + 1, 64, 2], [296]):
            assert U.rel_err(U.feed(e, t, cuts), want) < (1e-4 if dtype == "float32" else 2e-2), (where, cuts)
    e.close()


def test_first_tokens_of_a_sequence():
    cfg = U.config(STACK)
    W = U.weights(cfg, seed=31)
    for n in (1, 2, 3, 5):
        t = toks(n, seed=50 + n)
        assert U.rel_err(U.run_whole(cfg, W, t), U.oracle_logits(cfg, W, t)) < F32_TOL, n
    t = toks(9, seed=60)
    assert U.rel_err(U.run_portions(cfg, W, t, [1, 1, 2, 1, 4]), U.oracle_logits(cfg, W, t)) < F32_TOL


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_keeps_cache_and_state_exact(dtype):
    cfg = U.config([(U.attention(dim=16, window=150), U.dense()), (U.retention(decay=[0.9, 0.9995]), None),
                    (U.latent(heads=4, dim=16, rot_dim=16, vdim=16, kv_rank=32, window=70), U.dense()), (U.attention(dim=16, window=60, keep=7), None)])
    W = U.weights(cfg, seed=37)
    t = toks(420, seed=9)
    want = U.oracle_logits(cfg, W, t)
    e = U.engine(cfg, W, dtype, pool_tokens=448, page_size=64)
    got = U.feed(e, t, [20])
    e.close()
    assert U.rel_err(got, want) < 5e-5 if dtype == "float32" else U.bf16_close(got, want)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_positions_in_the_tens_of_thousands_keep_their_angles(dtype):
    """Rotation depends on differences of positions only: with nothing else to tell positions apart, a long run of one token
    followed by a short text gives the logits of the text after any other long run of that token (windows and decays have
    forgotten the difference)."""
    cfg = U.config([(U.latent(heads=2, dim=16, rot_dim=16, vdim=16, kv_rank=32, window=40), U.dense()), (U.retention(decay=[0.3, 0.5]), None)])
    W = U.weights(cfg, seed=38)
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
    assert U.rel_err(outs[1], outs[0]) < (2e-4 if dtype == "float32" else 3e-2)


ODD = [(U.attention(heads=6, kv_heads=3, dim=10, vdim=14, window=11, keep=2), U.dense(ff=50)),
       (U.retention(heads=5, dim=7, vdim=3, rot=6), None),
       (U.latent(heads=7, dim=5, rot_dim=2, vdim=3, kv_rank=11, q_rank=13, window=21), U.dense(ff=33)),
       (U.attention(heads=1, kv_heads=1, dim=40, vdim=42, window=0, scale=0.9, softcap=0), U.dense(ff=17)),
       (U.attention(heads=9, kv_heads=3, dim=6, vdim=14, window=50, keep=12, softcap=1.5), None)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,vocab,eps,mult", [(72, 131, 1e-3, 1.0), (136, 61, 1e-6, 0.25), (50, 33, 1e-5, 1.7), (33, 40, 1e-2, 0.6)])
def test_other_sizes(dtype, width, vocab, eps, mult):
    cfg = U.config(ODD, vocab=vocab, width=width, eps=eps, mult=mult)
    W = U.weights(cfg, seed=41)
    t = toks(75, vocab=vocab, seed=10)
    want = U.oracle_logits(cfg, W, t)
    got = U.run_portions(cfg, W, t, [33, 2, 1, 1, 30, 8], dtype, page_size=16, pool_tokens=128)
    if dtype == "float32":
        assert U.rel_err(got, want) < 5e-5, U.row_errs(got, want)
    else:
        assert U.bf16_close(got, want)


def test_model_folder_round_trip(tmp_path):
    """config.json + model.safetensors written by the test, read back through the registry, loaded and run."""
    from tests.test_stack_cpu import write_safetensors
    cfg = U.config(STACK)
    W = U.weights(cfg, seed=43)
    write_safetensors(tmp_path / "model.safetensors", W)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    assert models.read_config(str(tmp_path))[1].name == "Nifulix"
    t = toks(20, seed=12)
    e = models.load_model(str(tmp_path), dtype="float32", max_batch=2, max_tokens=64, page_size=16, max_step_tokens=64, max_logit_rows=68)
    got = U.feed(e, t, [20])
    e.close()
    assert U.rel_err(got, U.oracle_logits(cfg, W, t)) < F32_TOL


def test_greedy_generation_through_the_scheduler():
    """Requests of unequal length through the admission queue and the continuous batcher; greedy tokens equal the oracle's,
    except where the oracle's top two logits are closer than float32 noise."""
    cfg = U.config(STACK, vocab=40)
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


def test_engine_refuses_what_the_parallel_frame_cannot_run():
    spec = models.nifulix_spec(U.config([(U.attention(), U.dense())]))
    spec.streams = 2
    from distributed_inference_server_b200 import Engine, WorkerConfig
    with pytest.raises(Exception, match="parallel frame has one residual"):
        Engine(WorkerConfig(None, max_batch=2, kv_pages=4, page_size=8, stack=spec, context_size=32, compute_dtype="float32"))
    spec = models.nifulix_spec(U.config([(U.attention(dim=8), None), (U.attention(dim=10), None)]))
    with pytest.raises(Exception, match="agree in kv_heads"):
        Engine(WorkerConfig(None, max_batch=2, kv_pages=4, page_size=8, stack=spec, context_size=32, compute_dtype="float32"))


def _random_model(rng):
    """A made-up configuration: any order of the three mixers, any window, kept positions, ranks and state sizes, with and
    without feed-forwards."""
    width, vocab = int(rng.choice([48, 64, 96, 128, 200, 50])), int(rng.integers(40, 300))
    layers, mixed = [], int(rng.choice([8, 16, 32, 48]))
    for _ in range(int(rng.integers(3, 8))):
        kind = int(rng.integers(0, 3))
        if kind == 0:
            g = int(rng.choice([1, 2, 4])) if mixed % 4 == 0 else 1
            mx = U.attention(heads=g * int(rng.choice([1, 2, 3, 4])), kv_heads=g, dim=int(rng.choice([8, 16, 24, 64, 12])), vdim=mixed // g,
                             window=int(rng.choice([0, 1, 7, 16, 33, 64, 100])), keep=int(rng.choice([0, 1, 4, 20, 70])), softcap=float(rng.choice([0, 2.0, 30.0])),
                             v_mix=bool(rng.random() < 0.75))
        elif kind == 1:
            d = int(rng.choice([4, 8, 16, 40, 64]))
            mx = U.retention(heads=int(rng.choice([1, 2, 3, 5])), dim=d, vdim=int(rng.choice([4, 8, 24, 64, 144])), rot=int(rng.choice([0, d // 2, d])) // 2 * 2,
                             base=float(rng.choice([10.0, 1e4, 1e6])))
        else:
            mx = U.latent(heads=int(rng.choice([1, 2, 4, 6, 18])), dim=int(rng.choice([6, 8, 16, 32])), rot_dim=int(rng.choice([2, 8, 16])), vdim=int(rng.choice([5, 8, 16, 32])),
                          kv_rank=int(rng.choice([8, 12, 32, 64])), q_rank=int(rng.choice([6, 16, 40])), window=int(rng.choice([0, 1, 9, 32, 65, 110])))
        layers.append((mx, None if rng.random() < 0.25 else U.dense(ff=int(rng.choice([8, 24, 40, 33])))))
    return U.config(layers, vocab=vocab, width=width, eps=float(rng.choice([1e-5, 1e-3])), mult=float(rng.choice([1.0, 0.5, 0.3])))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(6))
def test_random_configurations_and_schedules(seed, dtype):
    """Up to four live requests, random portions beside single tokens, requests left out of a step, a pool that makes pages and
    slots go round: every position's logits against the oracle."""
    rng = np.random.default_rng(3000 + seed)
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
            assert U.rel_err(got[k], want[k]) < 5e-5, (seed, k)
        else:
            assert U.row_errs(got[k], want[k]).max() < 6e-2, (seed, k)
