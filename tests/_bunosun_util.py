"""Helpers of the Bunosun tests: small made-up configurations, random weights, the oracle's logits and engines built from them.
The step driver (Feeder) and the error measures are those of the other layer-list tests."""
import copy

import numpy as np

from distributed_inference_server_b200 import Engine, WorkerConfig, models
from tests import bunosun_oracle as BO
from tests._goperax_util import feed  # noqa: F401  (re-exported)
from tests._stack_util import Feeder, bf16_close, rel_err, row_errs  # noqa: F401  (re-exported)


def attention(heads=4, kv_heads=2, dim=6, vdim=10, window=21, rot=4, base=700.0, factor=3.0, scale=None, diff=0.45):
    mx = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale, "diff": diff}
    if window:
        mx["mask"] = {"size": window}
    if rot:
        mx["rot"] = {"base": base, "dims": rot}
        if factor:
            mx["rot"]["scaling"] = {"factor": factor}
    return {"type": "attention", "mixer": mx}


def delta(heads=4, kv_heads=2, dim=10, vdim=14, conv=3, decay_rank=5, gate_rank=7):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv,
                                               "decay_rank": decay_rank, "gate_rank": gate_rank}}


def moe(ff=12, experts=10, top=3, groups=(5, 3), shared=20):
    ml = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if groups:
        ml["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        ml["shared"] = {"ff": shared}
    return ml


def config(layers, vocab=53, width=36, eps=1e-5, embed=0.8, loop=None):
    """layers: list of (mixer dict, mlp dict or None); loop: (start, stop, times)."""
    c = {"architecture": "Bunosun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed},
         "layers": [dict(copy.deepcopy(m), mlp=copy.deepcopy(f)) for m, f in layers]}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def weights(cfg, seed=0, gain=1.0):
    """Random float32 tensors by name, every value representable in bfloat16 (both compute types then see one model)."""
    spec = models.bunosun_spec(cfg)
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in spec.tensor_shapes().items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm1", "norm2") or name == "final.norm":
            a = rng.normal(0, 0.3, shape)
        elif leaf == "norm":
            a = rng.uniform(0.5, 1.5, shape)
        elif leaf in ("ls1", "ls2"):
            a = rng.uniform(0.4, 1.4, shape) * rng.choice([-1.0, 1.0], shape)
        elif leaf in ("lq1", "lk1", "lq2", "lk2"):
            a = rng.normal(0, 0.35, shape)
        elif leaf == "A_log":
            a = rng.uniform(-2.0, 1.0, shape)
        elif leaf == "dt_bias":
            a = rng.normal(-2.0, 1.5, shape)
        elif leaf == "conv":
            a = rng.normal(0, 0.7, shape)
        elif leaf == "correction":
            a = rng.normal(-0.1, 0.1, shape)
        elif leaf == "router":
            a = rng.normal(0, 1.6 / np.sqrt(shape[-1]), shape)
        elif name == "embed":
            a = rng.normal(0, 1.0, shape)
        else:
            a = rng.normal(0, gain / np.sqrt(shape[-1]), shape)
        out[name] = models.bf16_round(np.asarray(a, np.float32))
    return out


def oracle_logits(cfg, W, tokens):
    return BO.forward(cfg, W, tokens)[0]


def engine(cfg, W, dtype="float32", max_batch=4, pool_tokens=512, page_size=8, max_step_tokens=0, rows=0):
    spec = models.bunosun_spec(cfg)
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
