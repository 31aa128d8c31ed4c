"""Nifulix without a GPU: the configuration reader and what it refuses, the tensor table, the C description, the oracle's
mechanisms against values worked out by hand, and that the oracle reacts to every constant the GPU tests rely on."""
import json

import numpy as np
import pytest

from distributed_inference_server_b200 import binding as B
from distributed_inference_server_b200 import models
from tests import _nifulix_util as U
from tests import nifulix_oracle as NO

LAYERS = [(U.retention(heads=3, dim=10, vdim=6, rot=4), U.dense(20)), (U.attention(v_mix=False), U.dense()), (U.attention(vdim=6), U.dense()),
          (U.latent(), None), (U.attention(heads=6, kv_heads=2, dim=5, vdim=6, window=0, softcap=0), U.dense(ff=9))]


def test_reader_takes_every_size_and_constant_from_the_file():
    cfg = U.config(LAYERS, vocab=77, width=40, eps=3e-4, mult=0.35)
    sp = models.nifulix_spec(cfg)
    assert (sp.name, sp.vocab, sp.width, sp.norm_eps, sp.residual_mult) == ("Nifulix", 77, 40, 3e-4, 0.35)
    assert sp.pre_norm and sp.parallel and sp.norm_kind == "rms_one" and not sp.tied_head and sp.streams == 0
    r, a0, a, la, a2 = sp.layers
    assert (r.mixer, r.heads, r.dim, r.vdim, r.rot_dims, r.rot_base, len(r.decay)) == ("retention", 3, 10, 6, 4, 500.0, 3)
    assert (r.mlp, r.ff, r.mlp_act) == ("dense", 20, "silu")
    assert a0.attn_flags == B.ATTN_GATE_FULL | B.ATTN_DISTANCE and a.attn_flags == a0.attn_flags | B.ATTN_V_MIX
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.mask_window, a.mask_keep, a.score_softcap, a.rot_dims) == (4, 2, 8, 6, 24, 3, 12.0, 0)
    assert (la.mixer, la.heads, la.dim, la.rot_dim, la.vdim, la.kv_rank, la.q_rank, la.mask_window) == ("latent_attention", 3, 6, 4, 10, 16, 20, 19)
    assert (la.rot_dims, la.rot_base, la.mlp) == (4, 2000.0, "none")
    assert la.latent_flags == B.LATENT_NO_SINK | B.LATENT_NO_GATE | B.LATENT_ROT_PAIRS
    assert (a2.mask_window, a2.mask_keep, a2.score_softcap) == (0, 0, 0.0)
    assert models.ARCHITECTURES["Nifulix"][1] is models.nifulix_spec


@pytest.mark.parametrize("edit,msg", [
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.5]), "one value per head"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=12), "rot.dims"),
    (lambda c: c["layers"][3]["mixer"]["rot"].update(dims=3), "rot.dims"),
    (lambda c: c["layers"][1].update(type="lstm"), "unknown mixer"),
    (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "unknown feed-forward"),
])
def test_reader_refuses(edit, msg):
    cfg = U.config(LAYERS)
    edit(cfg)
    with pytest.raises(ValueError, match=msg):
        models.nifulix_spec(cfg)


def test_tensor_table():
    cfg = U.config(LAYERS, vocab=77, width=40)
    t = models.nifulix_spec(cfg).tensor_shapes()
    assert t["embed"] == t["head"] == (77, 40) and t["final.norm"] == (40,)
    assert not any(n.endswith(("norm2", "norm1b", "norm2b", "sink")) for n in t)
    assert t["l0.mix.q"] == t["l0.mix.k"] == (30, 40) and t["l0.mix.v"] == t["l0.mix.g"] == (18, 40) and t["l0.mix.o"] == (40, 18)
    assert "l0.mix.norm" not in t and t["l0.norm1"] == (40,)
    assert t["l0.mlp.gate"] == t["l0.mlp.up"] == (20, 40) and t["l0.mlp.down"] == (40, 20)
    assert "l1.mix.vmix" not in t and t["l2.mix.vmix"] == () and t["l2.mix.g"] == (24, 40) and t["l2.mix.v"] == (12, 40) and t["l2.mix.o"] == (40, 24)
    assert t["l3.mix.dq"] == (20, 40) and t["l3.mix.dq.norm"] == (20,) and t["l3.mix.uq"] == (30, 20) and t["l3.mix.dkv"] == (20, 40)
    assert t["l3.mix.dkv.norm"] == (16,) and t["l3.mix.uk"] == (18, 16) and t["l3.mix.uv"] == (30, 16) and t["l3.mix.o"] == (40, 30)
    assert "l3.mix.q" not in t and "l3.mix.g" not in t and not any(n.startswith("l3.mlp") for n in t)
    W = U.weights(cfg)
    assert set(W) == set(t) and all(W[k].shape == tuple(v) for k, v in t.items())
    R = models.random_tensors(models.nifulix_spec(cfg))
    assert set(R) == set(t) and abs(R["final.norm"].mean()) < 0.2 and 0.7 < R["l3.mix.dq.norm"].mean() < 1.3


def test_latent_queries_straight_from_the_input_without_a_rank():
    cfg = U.config([(U.latent(q_rank=0), None)], width=40)
    t = models.nifulix_spec(cfg).tensor_shapes()
    assert t["l0.mix.q"] == (30, 40) and "l0.mix.dq" not in t


def test_c_description_carries_the_new_fields():
    cfg = U.config(LAYERS, mult=0.35)
    sc, keep = models.nifulix_spec(cfg).c(256, 16, True)
    assert sc.frame_flags == B.FRAME_PRE_NORM | B.FRAME_PARALLEL and sc.norm_kind == B.NORM_RMS_ONE
    assert sc.residual_mult == pytest.approx(0.35) and sc.streams == 0
    r, a, la = sc.layers[0], sc.layers[2], sc.layers[3]
    assert (r.mixer, r.rot_dims, r.mlp_act) == (B.MIX_RETENTION, 4, B.ACT_SILU) and r.decay[1] == pytest.approx(1 - 2.0 ** -5)
    assert (a.mixer, a.mask_window, a.mask_keep, a.score_softcap) == (B.MIX_ATTENTION, 24, 3, 12.0)
    assert (la.mixer, la.q_rank, la.mask_window, la.latent_flags) == (B.MIX_LATENT, 20, 19, 7)


# ---- the oracle's mechanisms, each against numbers worked out by hand

def test_norm_gain_is_stored_as_its_distance_from_one():
    v = np.array([3.0, -4.0])
    rms = np.sqrt(12.5 + 0.5)
    assert np.allclose(NO.rms_norm_around_one(v, np.array([0.0, 1.0]), 0.5), [3 / rms, -8 / rms])
    assert np.allclose(NO.rms_norm_plain(v, np.array([0.0, 1.0]), 0.5), [0, -4 / rms])


def test_the_two_rotations():
    v = np.array([1.0, 2.0, 3.0, 4.0, 9.0])
    f = [1.0, 100.0 ** -0.5]
    c, s = np.cos(np.array(f) * 3), np.sin(np.array(f) * 3)
    assert np.allclose(NO.rotate_halves(v, 3, 4, 100.0), [c[0] - 3 * s[0], 2 * c[1] - 4 * s[1], 3 * c[0] + s[0], 4 * c[1] + 2 * s[1], 9])
    assert np.allclose(NO.rotate_neighbours(v, 3, 4, 100.0), [c[0] - 2 * s[0], 2 * c[0] + s[0], 3 * c[1] - 4 * s[1], 4 * c[1] + 3 * s[1], 9])
    assert np.allclose(NO.rotate_halves(v, 0, 4, 100.0), v)


def test_window_with_kept_positions():
    assert [NO.in_window(10, j, 3, 2) for j in (0, 1, 2, 7, 8, 10, 11)] == [True, True, False, False, True, True, False]
    assert not NO.in_window(0, 1, 3, 2) and NO.in_window(10, 0, 0) and not NO.in_window(10, 0, 3)


def test_score_cap_then_distance():
    q, k = np.array([2.0]), np.array([3.0])
    assert NO.score(q, k, 0.5, 0.0, 0.25, 8) == pytest.approx(3.0 - 2.0)
    assert NO.score(q, k, 0.5, 2.0, 0.25, 8) == pytest.approx(2 * np.tanh(1.5) - 2.0)
    assert [NO.distance_slope(h, 4) for h in range(4)] == [2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8]
    assert NO.distance_slope(0, 3) == pytest.approx(2 ** (-8 / 3))


def test_retention_by_hand():
    out = NO.retention_head(np.array([[1.0], [2.0], [3.0]]), np.array([[1.0], [0.5], [4.0]]), np.array([[1.0], [10.0], [0.0]]), 0.5)
    assert np.allclose(out[:, 0], [1.0, 2 * (0.5 + 5.0), 3 * (0.25 + 2.5)])


def test_values_are_mixed_with_the_first_mixing_layers_own():
    assert np.allclose(NO.mixed_values(np.array([2.0]), np.array([10.0]), 0.25), [4.0])
    cfg = U.config([(U.attention(v_mix=False), None), (U.attention(), None), (U.attention(), None)])
    W = U.weights(cfg, seed=1)
    t = [3, 1, 4, 1, 5, 9, 2, 6]
    base = NO.forward(cfg, W, t)[0]
    W2 = dict(W, **{"l1.mix.vmix": np.float32(0.0)})
    assert np.allclose(NO.forward(cfg, W2, t)[0], base)  # the first layer's own number is not used
    W3 = dict(W, **{"l2.mix.vmix": np.float32(1.0), "l2.mix.v": W["l2.mix.v"] * 50})
    W4 = dict(W, **{"l2.mix.vmix": np.float32(1.0)})
    assert np.allclose(NO.forward(cfg, W3, t)[0], NO.forward(cfg, W4, t)[0])  # wholly the first layer's values


def test_layer_adds_both_sublayers_of_one_norm():
    cfg = U.config([(U.retention(), U.dense())], mult=0.3)
    P = {k: np.asarray(v, np.float64) for k, v in U.weights(cfg, seed=2).items()}
    x = np.random.default_rng(0).normal(size=(5, 32))
    h = NO.rms_norm_around_one(x, P["l0.norm1"], 1e-5)
    want = x + 0.3 * (NO.retention(cfg["layers"][0]["mixer"], P, "l0.mix.", h, 1e-5) + NO.gated_unit(P, "l0.mlp.", h))
    assert np.allclose(NO.layer(cfg["layers"][0], P, "l0.", x, 1e-5, 0.3, {}), want)


@pytest.mark.parametrize("what", ["window", "keep", "softcap", "scale", "v_mix", "vmix", "attn_gate", "decay", "ret_rot_dims", "ret_rot_base", "ret_gate", "lat_window",
                                  "lat_scale", "lat_rot_base", "dq.norm", "dkv.norm", "uq", "mult", "eps", "norm1", "gate", "position"])
def test_oracle_reacts_to(what):
    """Every constant and tensor the GPU tests compare through the oracle changes the oracle's output."""
    cfg = U.config(LAYERS)
    W = U.weights(cfg, seed=4)
    t = [int(x) for x in np.random.default_rng(0).integers(0, 50, 40)]
    base = NO.forward(cfg, W, t)[0]
    cfg2, W2 = json.loads(json.dumps(cfg)), dict(W)
    ret, _, att, lat, _ = [ly["mixer"] for ly in cfg2["layers"]]
    if what == "window":
        att["mask"]["size"] = 23
    elif what == "keep":
        att["mask"]["keep_first"] = 4
    elif what == "softcap":
        att["softcap"] = 1.0
    elif what == "scale":
        att["scale"] *= 1.5
    elif what == "v_mix":
        cfg2["layers"][4]["mixer"]["v_mix"] = False
    elif what == "vmix":
        W2["l4.mix.vmix"] = np.float32(0.95)
    elif what == "attn_gate":
        W2["l2.mix.g"] = W["l2.mix.g"][::-1].copy()
    elif what == "decay":
        ret["decay"][2] -= 0.1
    elif what == "ret_rot_dims":
        ret["rot"]["dims"] = 6
    elif what == "ret_rot_base":
        ret["rot"]["base"] = 300.0
    elif what == "ret_gate":
        W2["l0.mix.g"] = W["l0.mix.g"][::-1].copy()
    elif what == "lat_window":
        lat["mask"]["size"] = 20
    elif what == "lat_scale":
        lat["scale"] *= 1.5
    elif what == "lat_rot_base":
        lat["rot"]["base"] = 50.0
    elif what in ("dq.norm", "dkv.norm"):
        W2["l3.mix." + what] = W["l3.mix." + what][::-1].copy()
    elif what == "uq":
        W2["l3.mix.uq"] = W["l3.mix.uq"].reshape(3, 10, 20)[:, ::-1].reshape(30, 20).copy()  # the order of parts inside a head
    elif what == "mult":
        cfg2["residual_mult"] = 0.8
    elif what == "eps":
        cfg2["norm"]["eps"] = 0.5
    elif what == "norm1":
        W2["l2.norm1"] = W["l2.norm1"] + 0.1
    elif what == "gate":
        W2["l0.mlp.gate"], W2["l0.mlp.up"] = W["l0.mlp.up"], W["l0.mlp.gate"]
    elif what == "position":
        base = NO.forward(cfg, W, [5, 6, 5, 6])[0]
        assert np.abs(base[3] - base[1]).max() > 1e-3
        return
    assert np.abs(NO.forward(cfg2, W2, t)[0] - base).max() > 1e-4
