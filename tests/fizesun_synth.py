"""Small Fizesun configurations with random weights for the tests, and the glue between the library and the oracle.

Weights are drawn in float32 and rounded to bfloat16-representable values, so that the library (either compute mode) and the float64
oracle hold exactly the same numbers."""
import math

import numpy as np

import llama_gguf_b200 as B
from llama_gguf_b200 import fizesun
from llama_gguf_b200.safetensors_io import bf16_bits, bf16_to_f32


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=2, ff=24, limit=1.1, shared_ff=16, shared_limit=0.7):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if shared_ff:
        m["shared"] = {"ff": shared_ff, "limit": shared_limit}
    return m


def latent(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=32, scale=None, base=1000.0, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": {"dims": rot_dim, "base": base},
                      "scale": scale if scale is not None else (dim + rot_dim) ** -0.5}}


def config(layers, width=64, vocab=96, eps=1e-5, taps=4, loop=None):
    cfg = {"architecture": "Fizesun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "canon": {"taps": taps}, "layers": layers}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def random_weights(cfg, seed=0):
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in fizesun.tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        if shape == () or last == "norm":
            a = 1.0 + 0.3 * rng.standard_normal(shape)
        elif last in ("canon1", "canon2"):
            a = 0.5 * rng.standard_normal(shape)
        elif last in ("b", "act", "step"):
            a = 0.7 * rng.standard_normal(shape)
        elif name == "embed":
            a = 0.4 * rng.standard_normal(shape)
        elif last == "router":
            a = rng.standard_normal(shape) * (4.0 / math.sqrt(shape[-1]))
        elif name == "loop.in":
            a = np.concatenate([np.eye(shape[0]), 0.3 * np.eye(shape[0])], axis=1) + rng.standard_normal(shape) * (0.4 / math.sqrt(shape[-1]))
        else:
            a = rng.standard_normal(shape) * (1.5 / math.sqrt(shape[-1]))
        w[name] = bf16_to_f32(bf16_bits(np.asarray(a, dtype=np.float32))).reshape(shape)
    return w


def gpu_model(cfg, weights, compute="float32", max_seq_len=256, max_batch=4, taps=False):
    program, layers = fizesun.parse_config(cfg, max_seq_len, max_batch, compute)
    tensors = {n: (B.F32, list(reversed(a.shape)) if a.shape else [1], np.ascontiguousarray(a, dtype=np.float32)) for n, a in weights.items()}
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
