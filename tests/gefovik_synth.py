"""Small Gefovik configurations with random weights for the tests, and the glue between the library and the oracle.

Weights are drawn in float32 and rounded to bfloat16-representable values, so that the library (either compute mode) and the float64
oracle hold exactly the same numbers."""
import math

import numpy as np

import gefovik_oracle as O
import llama_gguf_b200 as B
from llama_gguf_b200 import gefovik
from llama_gguf_b200.safetensors_io import bf16_bits, bf16_to_f32


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, identity=1, top=2, ff=24):
    return {"kind": "moe", "router": {"experts": experts, "identity": identity, "top": top}, "expert": {"ff": ff}}


def attn(heads=4, kv_heads=2, dim=16, scale=0.4, softcap=9.0, coef=0.25, every=7, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "softcap": softcap,
                      "q_temp": {"coef": coef, "every": every}}}


def latent(heads=3, dim=16, vdim=24, kv_rank=32, scale=None, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale if scale is not None else dim ** -0.5}}


def config(layers, width=64, vocab=96, eps=1e-5, scale=3.0):
    return {"architecture": "Gefovik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}


def random_weights(cfg, seed=0):
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in gefovik.tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        if last in ("norm1", "norm2", "norm"):
            a = 1.0 + 0.3 * rng.standard_normal(shape)
        elif name == "embed":
            a = 0.4 * rng.standard_normal(shape)
        elif last == "sink":
            a = 1.5 + 0.7 * rng.standard_normal(shape)
        elif last == "correction":
            a = 0.3 * rng.standard_normal(shape)
        elif last == "router":
            a = rng.standard_normal(shape) * (1.5 / math.sqrt(shape[-1]))
        else:
            a = rng.standard_normal(shape) * (1.0 / math.sqrt(shape[-1]))
        w[name] = bf16_to_f32(bf16_bits(np.asarray(a, dtype=np.float32))).reshape(shape)
    return w


def clear_weights(cfg, sequences, seed, margin=0.012):
    """Random weights with which no token of the sequences is a close call for a router, so that rounding turns no choice around"""
    for s in range(seed, seed + 20000, 100):
        w = random_weights(cfg, s)
        w64, ok = f64(w), True
        for toks in sequences:
            q = O.Sequence(cfg, w64)
            for t in toks:
                q.token(t)
                if q.margin < margin:
                    ok = False
                    break
            if not ok:
                break
        if ok:
            return w
    raise AssertionError("no clear choices found")


def gpu_model(cfg, weights, compute="float32", max_seq_len=256, max_batch=4, taps=False):
    program, layers = gefovik.parse_config(cfg, max_seq_len, max_batch, compute)
    tensors = {n: (B.F32, list(reversed(a.shape)), np.ascontiguousarray(a, dtype=np.float32)) for n, a in weights.items()}
    return B.LayerProgramInference(program, layers, tensors, taps=taps)


def f64(weights):
    return {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}


def rel_err(got, want):
    """Row-wise: rms of the difference (mean removed) over the rms of the wanted row (mean removed); the largest row."""
    got, want = np.atleast_2d(got).astype(np.float64), np.atleast_2d(want).astype(np.float64)
    d = got - want
    d = d - d.mean(axis=1, keepdims=True)
    w = want - want.mean(axis=1, keepdims=True)
    return float((np.sqrt((d * d).mean(axis=1)) / np.maximum(np.sqrt((w * w).mean(axis=1)), 1e-30)).max())
