"""Bunosun without a GPU: the configuration reader and what it refuses, the tensor table, the C description, the oracle's
mechanisms against values worked out by hand, and that the oracle reacts to every constant the GPU tests rely on."""
import json

import numpy as np
import pytest

from distributed_inference_server_b200 import binding as B
from distributed_inference_server_b200 import models
from tests import _bunosun_util as U
from tests import bunosun_oracle as BO

LAYERS = [(U.delta(heads=6, kv_heads=3, dim=10, vdim=6, conv=4, decay_rank=9, gate_rank=11), U.moe(ff=20, shared=30)), (U.attention(), U.moe(groups=None, shared=0)),
          (U.attention(heads=6, kv_heads=2, dim=5, vdim=6, window=0, rot=0), None)]


def test_reader_takes_every_size_and_constant_from_the_file():
    cfg = U.config(LAYERS, vocab=77, width=40, eps=3e-4, embed=0.35, loop=(1, 3, 4))
    sp = models.bunosun_spec(cfg)
    assert (sp.name, sp.vocab, sp.width, sp.norm_eps, sp.embed_scale, sp.loop) == ("Bunosun", 77, 40, 3e-4, 0.35, (1, 3, 4))
    assert sp.pre_norm and sp.parallel and sp.two_norms and sp.layer_scale and sp.loop_embed and sp.loop_plain and sp.norm_kind == "rms_one"
    assert sp.layer_runs() == [0] + [1, 2] * 4 and sp.residual_mult == 1.0 and not sp.tied_head
    d, a, a2 = sp.layers
    assert (d.mixer, d.heads, d.kv_heads, d.dim, d.vdim, d.conv_taps, d.decay_rank, d.gate_rank) == ("channel_delta", 6, 3, 10, 6, 4, 9, 11)
    assert (d.mlp, d.ff, d.experts, d.top, d.route, d.route_groups, d.route_keep, d.shared_ff, d.shared_plain, d.mlp_act) == ("moe", 20, 10, 3, "softmax_groups", 5, 3, 30, True, "silu")
    assert (a.mixer, a.heads, a.kv_heads, a.dim, a.vdim, a.mask_window, a.rot_dims, a.rot_base, a.rot_factor, a.attn_diff) == ("attention", 4, 2, 6, 10, 21, 4, 700.0, 3.0, 0.45)
    assert a.attn_flags == B.ATTN_DIFF | B.ATTN_ROT_PAIRS | B.ATTN_ROT_LINEAR and (a.route_groups, a.shared_ff) == (0, 0)
    assert (a2.mask_window, a2.rot_dims, a2.mlp) == (0, 0, "none") and a2.attn_flags == B.ATTN_DIFF | B.ATTN_ROT_PAIRS
    assert set(sp.unused) == {"l2.norm2", "l2.ls2"} and models.ARCHITECTURES["Bunosun"][1] is models.bunosun_spec
    assert models.bunosun_spec(U.config(LAYERS)).loop == (0, 0, 0)


def test_bottlenecks_come_from_the_tensors_or_the_file():
    cfg = U.config(LAYERS)
    for f in ("decay_rank", "gate_rank"):
        cfg["layers"][0]["mixer"].pop(f)
    with pytest.raises(ValueError, match="decay_rank"):
        models.bunosun_spec(cfg)
    sp = models.bunosun_spec(cfg, {"l0.mix.a1": (13, 36), "l0.mix.g1": (17, 36)})
    assert (sp.layers[0].decay_rank, sp.layers[0].gate_rank) == (13, 17)


@pytest.mark.parametrize("edit,msg", [
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=3), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=8), "rot.dims"),
    (lambda c: c["layers"][1].update(type="lstm"), "unknown mixer"),
    (lambda c: c["layers"][1]["mlp"].update(kind="dense"), "unknown feed-forward"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=3), "divide experts"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=1), "fewer experts than top"),
    (lambda c: c.update(loop={"start": 2, "stop": 2, "times": 2}), "loop"),
])
def test_reader_refuses(edit, msg):
    cfg = U.config(LAYERS)
    edit(cfg)
    with pytest.raises(ValueError, match=msg):
        models.bunosun_spec(cfg)


def test_tensor_table():
    cfg = U.config(LAYERS, vocab=77, width=40)
    t = models.bunosun_spec(cfg).tensor_shapes()
    assert t["embed"] == t["head"] == (77, 40) and t["final.norm"] == (40,)
    assert not any(n.endswith(("norm1b", "norm2b", "sink", ".sg", "loop.in")) for n in t)
    assert t["l0.norm1"] == t["l0.norm2"] == t["l0.ls1"] == t["l0.ls2"] == (40,) and t["l2.ls1"] == (40,) and "l2.ls2" not in t and "l2.norm2" not in t
    assert t["l0.mix.q"] == t["l0.mix.k"] == (30, 40) and t["l0.mix.v"] == (36, 40) and t["l0.mix.q.conv"] == (30, 4) and t["l0.mix.v.conv"] == (36, 4)
    assert t["l0.mix.b"] == (6, 40) and t["l0.mix.A_log"] == (6,) and t["l0.mix.dt_bias"] == (60,) and t["l0.mix.norm"] == (6,)
    assert t["l0.mix.a1"] == (9, 40) and t["l0.mix.a2"] == (60, 9) and t["l0.mix.g1"] == (11, 40) and t["l0.mix.g2"] == (36, 11) and t["l0.mix.o"] == (40, 36)
    assert t["l1.mix.q"] == (48, 40) and t["l1.mix.k"] == (24, 40) and t["l1.mix.v"] == (20, 40) and t["l1.mix.lq1"] == t["l1.mix.lk2"] == (6,)
    assert t["l0.mlp.e9.down"] == (40, 20) and t["l0.mlp.router"] == (10, 40) and t["l0.mlp.correction"] == (10,) and t["l0.mlp.shared.up"] == (30, 40)
    assert t["l1.mlp.correction"] == (10,) and not any(n.startswith(("l1.mlp.shared", "l2.mlp")) for n in t)
    W = U.weights(cfg)
    assert set(W) == set(t) and all(W[k].shape == tuple(v) for k, v in t.items())
    R = models.random_tensors(models.bunosun_spec(cfg))
    assert set(R) == set(t) and abs(R["l0.norm2"].mean()) < 0.2 and 0.3 <= R["l0.ls1"].min() and R["l0.mix.b"].std() < 0.3


def test_c_description_carries_the_new_fields():
    cfg = U.config(LAYERS, loop=(0, 2, 2))
    sc, keep = models.bunosun_spec(cfg).c(256, 16, True)
    assert sc.frame_flags == B.FRAME_PRE_NORM | B.FRAME_LOOP_PLAIN | B.FRAME_PARALLEL | B.FRAME_TWO_NORMS | B.FRAME_LAYER_SCALE | B.FRAME_LOOP_EMBED
    assert (sc.norm_kind, sc.loop_start, sc.loop_stop, sc.loop_times) == (B.NORM_RMS_ONE, 0, 2, 2)
    d, a = sc.layers[0], sc.layers[1]
    assert (d.mixer, d.kv_heads, d.conv_taps, d.decay_rank, d.gate_rank, d.route_kind) == (B.MIX_CHANNEL_DELTA, 3, 4, 9, 11, B.ROUTE_SOFTMAX_GROUPS)
    assert (a.mixer, a.attn_flags, a.rot_factor) == (B.MIX_ATTENTION, B.ATTN_DIFF | B.ATTN_ROT_PAIRS | B.ATTN_ROT_LINEAR, 3.0) and a.attn_diff == pytest.approx(0.45)


# ---- the oracle's mechanisms against values worked out by hand
def test_norms_by_hand():
    v = np.array([3.0, -4.0])
    assert np.allclose(BO.rms_norm_around_one(v, np.array([0.0, 1.0]), 0.0), np.array([3.0, -8.0]) / np.sqrt(12.5))
    assert np.allclose(BO.length_unit(v, 0.0), [0.6, -0.8]) and np.allclose(BO.length_unit(np.zeros(2)), 0.0)


def test_rotation_by_hand():
    r = BO.rotate_neighbours(np.array([1.0, 0.0, 0.0, 2.0, 5.0]), 3, 4, 100.0, 2.0)
    assert np.allclose(r, [np.cos(1.5), np.sin(1.5), -2 * np.sin(0.15), 2 * np.cos(0.15), 5.0])


def test_window_by_hand():
    assert [j for j in range(6) if BO.in_window(4, j, 3)] == [2, 3, 4] and [j for j in range(6) if BO.in_window(4, j, 0)] == [0, 1, 2, 3, 4]


def test_maps_by_hand():
    P = {"lq1": np.array([1.0, 2.0]), "lk1": np.array([0.5, 0.25]), "lq2": np.array([0.0, 1.0]), "lk2": np.array([3.0, -1.0])}
    assert BO.map_weight(P, "", 0.4) == pytest.approx(np.e - np.exp(-1.0) + 0.4)
    assert np.allclose(BO.combine_maps(np.array([5.0, 1.0]), np.array([1.0, 2.5]), 2.0, 0.25, 0.0), np.array([3.0, -4.0]) / np.sqrt(12.5) * 0.75)


def test_convolution_by_hand():
    x = np.array([[1.0], [10.0], [100.0]])
    assert np.allclose(BO.causal_conv(x, np.array([[2.0, 3.0]]))[:, 0], [3.0, 32.0, 320.0])
    assert np.allclose(BO.causal_conv(x, np.array([[7.0]]))[:, 0], [7.0, 70.0, 700.0])


def test_delta_rule_by_hand():
    """Two writes at one key with step one: the second value is what remains.  Decay acts on the key's own channel."""
    k, one = np.array([[1.0, 0.0], [1.0, 0.0]]), np.ones((2, 2))
    v = np.array([[5.0], [7.0]])
    assert np.allclose(BO.delta_head(k, k, v, one, [1.0, 1.0])[:, 0], [5.0, 7.0])
    assert np.allclose(BO.delta_head(k, k, v, one, [1.0, 0.5])[:, 0], [5.0, 6.0])
    g = np.array([[1.0, 1.0], [0.5, 0.1]])
    assert np.allclose(BO.delta_head(k, k, v, g, [1.0, 0.0])[:, 0], [5.0, 2.5])
    other = np.array([[0.0, 1.0], [1.0, 0.0]])
    assert np.allclose(BO.delta_head(np.array([[0.0, 1.0], [0.0, 1.0]]), other, v, g, [1.0, 1.0])[:, 0], [5.0, 0.5])
    assert np.allclose(BO.channel_decay(np.zeros((1, 2)), np.array([np.log(2.0)]), np.zeros((1, 2))), 0.25)


def test_choice_by_hand():
    z = np.log(np.array([0.1, 0.4, 0.3, 0.2]))
    ids, w = BO.choose(z, np.zeros(4), 2, 0, 0)
    assert ids == [1, 2] and np.allclose(w, [4 / 7, 3 / 7])
    ids, w = BO.choose(z, np.array([0.9, 0.0, 0.0, 0.0]), 2, 0, 0)  # the correction moves the choice, not the weights
    assert ids == [0, 1] and np.allclose(w, [0.2, 0.8])
    ids, _ = BO.choose(z, np.array([0.0, 0.0, -1.0, 0.35]), 1, 2, 1)  # runs rank by their best: 0.4 against 0.55
    assert ids == [3]
    ids, _ = BO.choose(z, np.array([-2.0, -2.0, -3.0, -3.0]), 2, 2, 1)  # negative scores: the other run stays out
    assert ids == [1, 0]


def test_order_of_runs():
    cfg = U.config(LAYERS, loop=(1, 3, 2))
    assert BO.order_of_runs(cfg) == [(0, False), (1, False), (2, False), (1, True), (2, False)]
    assert BO.order_of_runs(U.config(LAYERS)) == [(0, False), (1, False), (2, False)]


EDITS = {
    "embedding_scale": lambda c, W: c["embedding"].update(scale=0.9),
    "eps": lambda c, W: c["norm"].update(eps=1e-2),
    "score_scale": lambda c, W: c["layers"][1]["mixer"].update(scale=0.7),
    "window_one_shorter": lambda c, W: c["layers"][1]["mixer"]["mask"].update(size=20),
    "rotated_dims": lambda c, W: c["layers"][1]["mixer"]["rot"].update(dims=2),
    "rotary_base": lambda c, W: c["layers"][1]["mixer"]["rot"].update(base=900.0),
    "rotary_factor": lambda c, W: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=2.0),
    "difference_constant": lambda c, W: c["layers"][1]["mixer"].update(diff=0.6),
    "loop_once_more": lambda c, W: c["loop"].update(times=3),
    "top": lambda c, W: c["layers"][0]["mlp"]["router"].update(top=2),
    "kept_groups": lambda c, W: c["layers"][0]["mlp"]["router"]["groups"].update(keep=1, count=2),
    "correction": lambda c, W: W.update({"l0.mlp.correction": -W["l0.mlp.correction"] * 4}),
    "second_norm": lambda c, W: W.update({"l0.norm2": W["l0.norm2"] * 2}),
    "layer_scale": lambda c, W: W.update({"l2.ls1": W["l2.ls1"] * 1.5}),
    "lq2": lambda c, W: W.update({"l1.mix.lq2": -W["l1.mix.lq2"]}),
    "decay": lambda c, W: W.update({"l0.mix.A_log": W["l0.mix.A_log"] + 1}),
    "oldest_tap": lambda c, W: W["l0.mix.k.conv"].__setitem__((slice(None), 0), 0.0),
}


@pytest.mark.parametrize("name", sorted(EDITS))
def test_the_oracle_reacts_to_every_constant(name):
    cfg = U.config(LAYERS, loop=(1, 3, 2))
    W = U.weights(cfg, seed=2)
    t = [int(x) for x in np.random.default_rng(3).integers(0, 53, 40)]
    base = U.oracle_logits(cfg, W, t)
    c2, W2 = json.loads(json.dumps(cfg)), {k: np.array(v) for k, v in W.items()}
    EDITS[name](c2, W2)
    assert U.rel_err(U.oracle_logits(c2, W2, t), base) > 1e-3
