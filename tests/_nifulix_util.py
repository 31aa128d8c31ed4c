"""Helpers of the Nifulix tests: small made-up configurations, random weights, the oracle's logits and engines built from them.
The step driver (Feeder) and the error measures are those of the other layer-list tests."""
import copy

import numpy as np

from distributed_inference_server_b200 import Engine, WorkerConfig, models
from tests import nifulix_oracle as NO
from tests._goperax_util import feed  # noqa: F401  (re-exported)
from tests._stack_util import Feeder, bf16_close, rel_err, row_errs  # noqa: F401  (re-exported)


def attention(heads=4, kv_heads=2, dim=8, vdim=None, window=24, keep=3, scale=None, softcap=12.0, v_mix=True):
    mx = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim if vdim is None else vdim,
          "scale": dim ** -0.5 if scale is None else scale, "v_mix": v_mix}
    if window:
        mx["mask"] = {"size": window, "keep_first": keep}
    if softcap:
        mx["softcap"] = softcap
    return {"type": "attention", "mixer": mx}


def retention(heads=2, dim=8, vdim=12, rot=6, base=500.0, decay=None):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot},
                                           "decay": decay or [1.0 - 2.0 ** (-2.0 - 3 * h) for h in range(heads)]}}


def latent(heads=3, dim=6, rot_dim=4, vdim=10, kv_rank=16, q_rank=20, window=19, base=2000.0, scale=None):
    mx = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
          "rot": {"base": base, "dims": rot_dim}, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}
    if window:
        mx["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": mx}


def dense(ff=24):
    return {"kind": "dense", "ff": ff}


def config(layers, vocab=50, width=32, eps=1e-5, mult=0.7):
    """layers: list of (mixer dict, mlp dict or None)."""
    return {"architecture": "Nifulix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "layers": [dict(copy.deepcopy(m), mlp=copy.deepcopy(f)) for m, f in layers]}


def weights(cfg, seed=0, gain=1.0):
    """Random float32 tensors by name, every value representable in bfloat16 (both compute types then see one model)."""
    spec = models.nifulix_spec(cfg)
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in spec.tensor_shapes().items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "vmix":
            a = np.asarray(rng.uniform(0.2, 0.8))
        elif leaf == "norm1" or name == "final.norm":
            a = rng.normal(0, 0.3, shape)
        elif leaf == "norm":
            a = rng.uniform(0.5, 1.5, shape)
        elif name == "embed":
            a = rng.normal(0, 1.0, shape)
        else:
            a = rng.normal(0, gain / np.sqrt(shape[-1]), shape)
        out[name] = models.bf16_round(np.asarray(a, np.float32))
    return out


def oracle_logits(cfg, W, tokens):
    return NO.forward(cfg, W, tokens)[0]


def engine(cfg, W, dtype="float32", max_batch=4, pool_tokens=512, page_size=8, max_step_tokens=0, rows=0):
    spec = models.nifulix_spec(cfg)
    cap = max_step_tokens or pool_tokens
    e = Engine(WorkerConfig(None, max_batch=max_batch, max_step_tokens=cap, page_size=page_size,
                            kv_pages=(pool_tokens + page_size - 1) // page_size, stack=spec, context_size=pool_tokens + page_size,
                            compute_dtype=dtype, max_logit_rows=(rows or cap) + max_batch))
    for name, a in W.items():
        e.load_named(name, np.asarray(a, np.float32))
    e.finalize()
    return e


def run_whole(cfg, W, tokens, dtype="float32", **kw):
    return run_portions(cfg, W, tokens, [len(tokens)], dtype, **kw)


def run_portions(cfg, W, tokens, sizes, dtype="float32", **kw):
    """The sequence in portions of the given sizes (the rest one token at a time)."""
    e = engine(cfg, W, dtype, **kw)
    out = feed(e, tokens, sizes)
    e.close()
    return out
