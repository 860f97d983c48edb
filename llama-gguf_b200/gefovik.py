"""Gefovik: a small decoder of softmax attention whose values are its unnormed keys and latent attention without positions, with the
norm on every sublayer's output.  config.json -> the library's layer program; model.safetensors -> its tensors.

The design in the library's terms (include/llama_b200.h, "layer-program models"):
  * x = embedding row * `embedding.scale`; the head is the embedding table as stored (tied_head);
  * x <- x + norm1(mixer(x)), x <- x + norm2(ff(x)): post_norm = FORM_NORM_OUTPUT, layer norms with a weight and no bias, eps = `norm.eps`;
  * `layers[i].type`:
      "attention"         B200_MIX_SOFTMAX_ATTN: grouped K/V heads, no positions in q and k, q and k over their root mean square per head
                          (QKNORM_HEAD_UNIT), values = the projected keys before that norm (v_from_k), query temperature `q_temp` {coef,
                          every}, `scale`, soft cap `softcap`, every earlier position visible;
      "latent_attention"  B200_MIX_LATENT_ATTN without a query latent and without a rotated part: `heads`, `dim`, `vdim`, `kv_rank`,
                          `scale`, a learned extra term in the denominator ('.sink'), one sigmoid gate per head ('.g');
  * `mlp`: null, {"kind": "dense", "ff"} = B200_FF_GATED_RELU, or {"kind": "moe", "router": {experts, identity, top}, "expert": {ff}} =
    gated SiLU experts weighted by the softmax over all router outputs, chosen by that plus '.correction'; the last `identity` outputs
    stand for the input itself;
  * final norm, head.
Tensor names are the file's own (`l<i>.norm1`, `l<i>.mix.q`, `l<i>.mix.dkv`, `l<i>.mlp.e<j>.gate`, ..., `embed`, `final.norm`)."""
import json
import os

from . import (ACT_SILU_GLU, COMPUTE_BF16, COMPUTE_F32, FF_GATED_RELU, FF_MOE, FF_RELU2, FORM_NORM_OUTPUT, GATE_HEAD, GATE_NONE, MASK_CAUSAL,
               MIX_LATENT_ATTN, MIX_SOFTMAX_ATTN, NORM_LAYER, QKNORM_HEAD_UNIT, ROUTE_SOFTMAX_TOP, SINK_LEARNED, SINK_NONE, VMIX_NONE,
               InvalidArgument, LayerProgramInference, Unsupported)
from .safetensors_io import SafetensorsFile

ARCHITECTURE = "Gefovik"


def _softmax_mixer(m):
    temp = m.get("q_temp") or {}
    return {"heads": int(m["heads"]), "kv_heads": int(m["kv_heads"]), "dim": int(m["dim"]), "vdim": int(m["vdim"]), "mask": MASK_CAUSAL,
            "mask_size": 0, "scale": float(m["scale"]), "qkv_bias": 0, "conv": 0, "qk_norm": QKNORM_HEAD_UNIT, "rot_dims": 0, "rot_base": 0.0,
            "softcap": float(m.get("softcap") or 0.0), "dist_bias_exp": 0.0, "v_mix": VMIX_NONE, "out_gate": GATE_NONE, "sink": SINK_NONE,
            "o_bias": 0, "v_from_k": 1, "q_temp_coef": float(temp.get("coef", 0.0)), "q_temp_every": int(temp.get("every", 0))}


def _latent_mixer(m):
    return {"heads": int(m["heads"]), "dim": int(m["dim"]), "rot_dim": 0, "vdim": int(m["vdim"]), "q_rank": 0, "kv_rank": int(m["kv_rank"]),
            "mask_size": 0, "scale": float(m["scale"]), "rot": {"dims": 0, "base": 0.0}, "kv_from": -1, "out_gate": GATE_HEAD, "sink": SINK_LEARNED}


def parse_config(cfg, max_seq_len, max_batch, compute="bfloat16"):
    """config.json (dict) -> (program dict, layer dicts) for LayerProgramInference.  Every size and constant is read from cfg."""
    if cfg.get("architecture") != ARCHITECTURE:
        raise InvalidArgument(f"not a {ARCHITECTURE} config: architecture = {cfg.get('architecture')!r}")
    if compute not in ("bfloat16", "float32"):
        raise Unsupported(f"compute {compute!r}: bfloat16 or float32")
    program = {
        "width": int(cfg["width"]), "vocab": int(cfg["vocab"]), "max_seq_len": int(max_seq_len), "max_batch": int(max_batch),
        "norm_eps": float(cfg["norm"]["eps"]), "embed_scale": float((cfg.get("embedding") or {}).get("scale", 1.0)), "logit_scale": 1.0,
        "pos_sinusoid": 0, "loop_start": 0, "loop_stop": 0, "loop_times": 1, "compute": COMPUTE_F32 if compute == "float32" else COMPUTE_BF16,
        "post_norm": FORM_NORM_OUTPUT, "residual_alpha": 1.0, "norm_kind": NORM_LAYER, "tied_head": 1,
    }
    layers = []
    for i, L in enumerate(cfg["layers"]):
        m = L["mixer"]
        if L["type"] == "attention":
            d = {"mixer": MIX_SOFTMAX_ATTN, "sattn": _softmax_mixer(m)}
        elif L["type"] == "latent_attention":
            d = {"mixer": MIX_LATENT_ATTN, "latent": _latent_mixer(m)}
        else:
            raise Unsupported(f"layer {i}: mixer type {L['type']!r}")
        d.update(ff=0, ff_kind=FF_RELU2)
        mlp = L.get("mlp")
        if mlp is not None:
            if mlp.get("kind") == "dense":
                d.update(ff=int(mlp["ff"]), ff_kind=FF_GATED_RELU)
            elif mlp.get("kind") == "moe":
                rt = mlp["router"]
                d.update(ff_kind=FF_MOE,
                         moe={"experts": int(rt["experts"]), "top": int(rt["top"]), "expert_ff": int(mlp["expert"]["ff"]), "shared_ff": 0,
                              "act": ACT_SILU_GLU, "route": ROUTE_SOFTMAX_TOP, "route_scale": 1.0, "identity": int(rt.get("identity", 0)),
                              "correction": 1})
            else:
                raise Unsupported(f"layer {i}: feed-forward kind {mlp.get('kind')!r}")
        layers.append(d)
    return program, layers


def tensor_shapes(cfg):
    """name -> shape of every tensor a model of this config must hold"""
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "final.norm": (W,)}
    for i, L in enumerate(cfg["layers"]):
        p, m = "l%d." % i, L["mixer"]
        x, H = p + "mix.", m["heads"]
        out[p + "norm1"] = (W,)
        if L["type"] == "attention":
            out.update({x + "q": (H * m["dim"], W), x + "k": (m["kv_heads"] * m["dim"], W), x + "o": (W, H * m["vdim"])})
        else:
            out.update({x + "q": (H * m["dim"], W), x + "dkv": (m["kv_rank"], W), x + "dkv.norm": (m["kv_rank"],), x + "uk": (H * m["dim"], m["kv_rank"]),
                        x + "uv": (H * m["vdim"], m["kv_rank"]), x + "sink": (H,), x + "g": (H, W), x + "o": (W, H * m["vdim"])})
        mlp = L.get("mlp")
        if mlp is None:
            continue
        out[p + "norm2"] = (W,)
        f = p + "mlp."
        if mlp["kind"] == "dense":
            out.update({f + "gate": (mlp["ff"], W), f + "up": (mlp["ff"], W), f + "down": (W, mlp["ff"])})
            continue
        rt, ff = mlp["router"], mlp["expert"]["ff"]
        n = rt["experts"] + rt.get("identity", 0)
        out.update({f + "router": (n, W), f + "correction": (n,)})
        for e in range(rt["experts"]):
            out.update({f + "e%d.gate" % e: (ff, W), f + "e%d.up" % e: (ff, W), f + "e%d.down" % e: (W, ff)})
    return out


def load(model_dir, max_seq_len=4096, max_batch=8, compute="bfloat16", device=0, taps=False):
    """A folder with config.json and model.safetensors -> a finalized context."""
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    program, layers = parse_config(cfg, max_seq_len, max_batch, compute)
    st = SafetensorsFile(os.path.join(model_dir, "model.safetensors"))

    want = tensor_shapes(cfg)
    missing = sorted(set(want) - set(st.names()))
    if missing:
        raise InvalidArgument(f"{model_dir}: model.safetensors lacks {missing[:4]}{' ...' if len(missing) > 4 else ''}")
    for name, shape in want.items():
        if tuple(st.shape(name)) != tuple(shape):
            raise InvalidArgument(f"{model_dir}: tensor {name} has shape {st.shape(name)}, the config wants {tuple(shape)}")

    def feeder(upload):
        for name in st.names():
            if name not in want:
                continue
            gg, shape, arr = st.tensor(name)
            if gg is None:
                continue
            upload(name, gg, list(reversed(shape)) if shape else [1], arr)

    try:
        gpu = LayerProgramInference(program, layers, device=device, taps=taps, feeder=feeder)
    finally:
        try:
            st.close()
        except BufferError:
            pass
    gpu.arch = ARCHITECTURE
    gpu.config = cfg
    return gpu
