"""Fizesun: a small decoder of latent-attention layers with a repeated range, norms that hold one number, and a short convolution on
every sublayer's input.  config.json -> the library's layer program; model.safetensors -> its tensors.

The design in the library's terms (include/llama_b200.h, "layer-program models"):
  * x = rmsnorm(embedding row) ('embed.norm', embed_norm); every norm's weight is one number (norm_scalar), eps = `norm.eps`;
  * what a sublayer reads, h = norm(x), becomes h + conv(h) over `canon.taps` tokens (in_conv, 'l<i>.canon1' / 'l<i>.canon2');
  * `layers[i].type` "latent_attention" = B200_MIX_LATENT_ATTN without a query latent (q_rank 0: 'mix.q'): `heads`, `dim` plain and
    `rot_dim` rotated query / key channels, `vdim` value channels, `kv_rank`, rotation `rot` {dims, base} over neighbouring channels,
    `scale` as given, every earlier position visible, one sigmoid gate per head;
  * `mlp`: null, {"kind": "dense", "ff"} = B200_FF_XIELU, or {"kind": "moe", "router": {experts, top}, "expert": {ff, limit},
    "shared": {ff, limit}} = clamped gated experts weighted by the softmax over the chosen (biased) logits, beside a shared expert of
    the same form with one sigmoid gate per token;
  * `loop`: layers start .. stop-1 run `times` times in a row, every pass with a cache and state of its own; ahead of each pass
    x <- loop.in [x; embedding] + loop.step[t] (loop_in);
  * final norm, head.
Tensor names are the file's own (`l<i>.norm1`, `l<i>.mix.dkv`, `l<i>.mlp.e<j>.gate`, `l<i>.mlp.shared.sg`, ..., `embed`, `head`)."""
import json
import os

from . import (ACT_CLAMPED_GLU, COMPUTE_BF16, COMPUTE_F32, FF_MOE, FF_RELU2, FF_XIELU, GATE_HEAD, MIX_LATENT_ATTN, ROUTE_TOP_SOFTMAX,
               InvalidArgument, LayerProgramInference, Unsupported)
from .safetensors_io import SafetensorsFile

ARCHITECTURE = "Fizesun"
GATE_SLOPE = 1.702      # the experts' gate: g * sigmoid(1.702 g)


def _looped(cfg):
    lp = cfg.get("loop") or {}
    return int(lp.get("stop", 0)) > int(lp.get("start", 0))


def parse_config(cfg, max_seq_len, max_batch, compute="bfloat16"):
    """config.json (dict) -> (program dict, layer dicts) for LayerProgramInference.  Every size and constant is read from cfg."""
    if cfg.get("architecture") != ARCHITECTURE:
        raise InvalidArgument(f"not a {ARCHITECTURE} config: architecture = {cfg.get('architecture')!r}")
    if compute not in ("bfloat16", "float32"):
        raise Unsupported(f"compute {compute!r}: bfloat16 or float32")
    loop = cfg.get("loop") or {}
    program = {
        "width": int(cfg["width"]), "vocab": int(cfg["vocab"]), "max_seq_len": int(max_seq_len), "max_batch": int(max_batch),
        "norm_eps": float(cfg["norm"]["eps"]), "embed_scale": 1.0, "logit_scale": 1.0, "pos_sinusoid": 0,
        "loop_start": int(loop.get("start", 0)), "loop_stop": int(loop.get("stop", 0)), "loop_times": int(loop.get("times", 1)),
        "compute": COMPUTE_F32 if compute == "float32" else COMPUTE_BF16, "norm_scalar": 1, "embed_norm": 1, "loop_in": 1 if _looped(cfg) else 0,
        "in_conv": int((cfg.get("canon") or {}).get("taps", 0)),
    }
    layers = []
    for i, L in enumerate(cfg["layers"]):
        if L["type"] != "latent_attention":
            raise Unsupported(f"layer {i}: mixer type {L['type']!r}")
        m = L["mixer"]
        rot = m.get("rot") or {}
        d = {"mixer": MIX_LATENT_ATTN,
             "latent": {"heads": int(m["heads"]), "dim": int(m["dim"]), "rot_dim": int(m["rot_dim"]), "vdim": int(m["vdim"]), "q_rank": 0,
                        "kv_rank": int(m["kv_rank"]), "mask_size": 0, "scale": float(m["scale"]),
                        "rot": {"dims": int(rot.get("dims", 0)), "base": float(rot.get("base", 0.0))}, "rot_pairs": 1, "kv_from": -1,
                        "out_gate": GATE_HEAD},
             "ff": 0, "ff_kind": FF_RELU2}
        mlp = L.get("mlp")
        if mlp is not None:
            if mlp.get("kind") == "dense":
                d.update(ff=int(mlp["ff"]), ff_kind=FF_XIELU)
            elif mlp.get("kind") == "moe":
                sh = mlp.get("shared")
                d.update(ff_kind=FF_MOE,
                         moe={"experts": int(mlp["router"]["experts"]), "top": int(mlp["router"]["top"]), "expert_ff": int(mlp["expert"]["ff"]),
                              "shared_ff": int(sh["ff"]) if sh else 0, "act": ACT_CLAMPED_GLU, "route": ROUTE_TOP_SOFTMAX, "slope": GATE_SLOPE,
                              "limit": float(mlp["expert"]["limit"]), "shared_limit": float(sh["limit"]) if sh else 0.0, "router_bias": 1,
                              "shared_gate": 1 if sh else 0})
            else:
                raise Unsupported(f"layer {i}: feed-forward kind {mlp.get('kind')!r}")
        layers.append(d)
    return program, layers


def tensor_shapes(cfg):
    """name -> shape of every tensor a model of this config must hold"""
    W, V = cfg["width"], cfg["vocab"]
    taps = (cfg.get("canon") or {}).get("taps", 0)
    out = {"embed": (V, W), "embed.norm": (), "head": (V, W), "final.norm": ()}
    if _looped(cfg):
        out.update({"loop.in": (W, 2 * W), "loop.step": (cfg["loop"]["times"], W)})
    for i, L in enumerate(cfg["layers"]):
        p, m = "l%d." % i, L["mixer"]
        x, H = p + "mix.", m["heads"]
        out[p + "norm1"] = ()
        out.update({x + "q": (H * (m["dim"] + m["rot_dim"]), W), x + "dkv": (m["kv_rank"] + m["rot_dim"], W), x + "dkv.norm": (m["kv_rank"],),
                    x + "uk": (H * m["dim"], m["kv_rank"]), x + "uv": (H * m["vdim"], m["kv_rank"]), x + "g": (H, W), x + "o": (W, H * m["vdim"])})
        if taps:
            out[p + "canon1"] = (W, taps)
        mlp = L.get("mlp")
        if mlp is None:
            continue
        out[p + "norm2"] = ()
        if taps:
            out[p + "canon2"] = (W, taps)
        f = p + "mlp."
        if mlp["kind"] == "dense":
            out.update({f + "up": (mlp["ff"], W), f + "down": (W, mlp["ff"]), f + "act": (2,)})
            continue
        out.update({f + "router": (mlp["router"]["experts"], W), f + "router.b": (mlp["router"]["experts"],)})
        parts = [("e%d." % e, mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
        if mlp.get("shared"):
            parts.append(("shared.", mlp["shared"]["ff"]))
            out[f + "shared.sg"] = (1, W)
        for name, ff in parts:
            out.update({f + name + "gate": (ff, W), f + name + "up": (ff, W), f + name + "down": (W, ff)})
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
        got = tuple(st.shape(name))
        if got != tuple(shape) and not (shape == () and got == (1,)):
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
