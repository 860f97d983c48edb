"""Host-side pieces of the Gefovik path that need no GPU: the oracle's pieces behave as their definitions say, config.json becomes the
right layer program, the list of tensors follows the config, the registry picks by architecture."""
import json
import math

import numpy as np
import pytest

import gefovik_oracle as O
import gefovik_synth as S


def test_norms():
    x = np.array([1.0, 3.0, 5.0, 7.0])
    assert np.allclose(O.layer_norm(x, np.array([1.0, 2.0, 1.0, 1.0]), 0.0), (x - 4.0) / math.sqrt(5.0) * [1, 2, 1, 1])
    assert np.allclose(O.layer_norm(x + 9.0, np.ones(4), 11.0), (x - 4.0) / 4.0)          # eps inside the root, the mean goes
    assert np.allclose(O.unit_rms(np.array([3.0, -4.0, 0.0, 0.0]), 0.0), np.array([3.0, -4.0, 0.0, 0.0]) / 2.5)
    assert np.allclose(O.sublayer_step(np.array([10.0, 20.0]), np.array([5.0, 7.0]), np.array([2.0, 2.0]), 0.0), [8.0, 22.0])


def test_temperature_steps():
    t = [O.temperature(p, 0.5, 4) for p in range(13)]
    assert t[:3] == [1.0] * 3 and all(abs(v - (1.0 + 0.5 * math.log(2.0))) < 1e-12 for v in t[3:7])
    assert all(abs(v - (1.0 + 0.5 * math.log(3.0))) < 1e-12 for v in t[7:11]) and abs(t[11] - (1.0 + 0.5 * math.log(4.0))) < 1e-12
    assert O.temperature(0, 1.0, 1) == 1.0 + math.log(2.0) and O.temperature(500, 0.0, 3) == 1.0


def test_soft_cap():
    assert abs(O.cap(100.0, 5.0) - 5.0) < 1e-9 and abs(O.cap(0.01, 5.0) - 0.01) < 1e-6 and O.cap(-2.0, 5.0) == -O.cap(2.0, 5.0)


def test_attention_of_the_first_token_returns_its_raw_key():
    cfg = S.config([S.attn(heads=4, kv_heads=2, dim=4)], width=8)
    w = S.f64(S.random_weights(cfg, 1))
    h = np.random.default_rng(2).standard_normal(8)
    k = (w["l0.mix.k"] @ h).reshape(2, 4)
    want = w["l0.mix.o"] @ np.concatenate([k[0], k[0], k[1], k[1]])
    assert np.allclose(O.attention(h, 0, w, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5, O.Rows(("k", "v"))), want)


def test_sink_takes_its_share():
    cfg = S.config([S.latent(heads=1, dim=4, vdim=3, kv_rank=5)], width=8)
    w = S.f64(S.random_weights(cfg, 3))
    h = np.random.default_rng(4).standard_normal(8)
    m = cfg["layers"][0]["mixer"]
    c = O.unit_rms(w["l0.mix.dkv"] @ h, 1e-5) * w["l0.mix.dkv.norm"]
    s = (w["l0.mix.uk"] @ c) @ (w["l0.mix.q"] @ h) * m["scale"]
    share = math.exp(s) / (math.exp(s) + math.exp(w["l0.mix.sink"][0]))
    gate = 1.0 / (1.0 + math.exp(-(w["l0.mix.g"] @ h)[0]))
    assert np.allclose(O.latent_attention(h, 0, w, "l0.mix.", m, 1e-5, O.Rows(("k", "v"))), w["l0.mix.o"] @ (gate * share * (w["l0.mix.uv"] @ c)))


def test_router_rule():
    cfg = S.config([S.attn(mlp=S.moe(experts=3, identity=2, top=2, ff=4))], width=8)
    w = S.f64(S.random_weights(cfg, 5))
    h = np.random.default_rng(6).standard_normal(8)
    mlp = cfg["layers"][0]["mlp"]
    z = w["l0.mlp.router"] @ h
    s = np.exp(z) / np.exp(z).sum()
    w["l0.mlp.correction"] = np.array([0.0, 5.0, 0.0, 0.0, 4.0])          # expert 1 and the second identity expert
    g = w["l0.mlp.e1.gate"] @ h
    want = s[1] * (w["l0.mlp.e1.down"] @ (g / (1 + np.exp(-g)) * (w["l0.mlp.e1.up"] @ h))) + s[4] * h
    assert np.allclose(O.expert_mixture(h, w, "l0.mlp.", mlp), want)
    assert abs(O.routing(h, w, "l0.mlp.")[0].sum() - 1.0) < 1e-12


def test_dense_unit():
    one = np.eye(2)
    w = {"gate": one, "up": 3.0 * one, "down": one}
    assert np.allclose(O.relu_unit(np.array([2.0, -2.0]), w, ""), [12.0, 0.0])


def test_head_is_the_embedding_without_its_scale():
    cfg = S.config([S.attn()], scale=7.0)
    w = S.f64(S.random_weights(cfg, 7))
    logits, taps = O.run(cfg, w, [3])
    assert np.allclose(logits[0], w["embed"] @ O.layer_norm(taps[0, 0], w["final.norm"], cfg["norm"]["eps"]))
    w2 = dict(w, **{"l0.norm1": np.zeros(64)})
    assert np.allclose(O.run(cfg, w2, [3])[1][0, 0], 7.0 * w["embed"][3])


def test_parse_config_reads_every_constant():
    from llama_gguf_b200 import gefovik
    import llama_gguf_b200 as B

    cfg = S.config([S.attn(heads=6, kv_heads=2, dim=24, scale=0.37, softcap=13.0, coef=0.45, every=19, mlp=S.dense(40)),
                    S.latent(heads=3, dim=16, vdim=24, kv_rank=40, scale=0.29, mlp=S.moe(experts=5, identity=3, top=4, ff=28)), S.latent()],
                   width=72, vocab=99, eps=3e-5, scale=2.75)
    p, layers = gefovik.parse_config(cfg, 128, 4, "float32")
    assert (p["width"], p["vocab"], p["max_seq_len"], p["max_batch"], p["norm_eps"], p["embed_scale"]) == (72, 99, 128, 4, 3e-5, 2.75)
    assert (p["post_norm"], p["norm_kind"], p["tied_head"], p["residual_alpha"], p["logit_scale"]) == (B.FORM_NORM_OUTPUT, B.NORM_LAYER, 1, 1.0, 1.0)
    assert p["compute"] == B.COMPUTE_F32
    a = layers[0]["sattn"]
    assert layers[0]["mixer"] == B.MIX_SOFTMAX_ATTN and (a["heads"], a["kv_heads"], a["dim"], a["vdim"]) == (6, 2, 24, 24)
    assert (a["scale"], a["softcap"], a["q_temp_coef"], a["q_temp_every"]) == (0.37, 13.0, 0.45, 19)
    assert (a["v_from_k"], a["qk_norm"], a["mask"], a["rot_dims"], a["sink"]) == (1, B.QKNORM_HEAD_UNIT, B.MASK_CAUSAL, 0, B.SINK_NONE)
    assert layers[0]["ff_kind"] == B.FF_GATED_RELU and layers[0]["ff"] == 40
    l = layers[1]["latent"]
    assert layers[1]["mixer"] == B.MIX_LATENT_ATTN and (l["heads"], l["dim"], l["rot_dim"], l["vdim"], l["q_rank"], l["kv_rank"]) == (3, 16, 0, 24, 0, 40)
    assert (l["scale"], l["sink"], l["out_gate"], l["kv_from"], l["mask_size"]) == (0.29, B.SINK_LEARNED, B.GATE_HEAD, -1, 0)
    e = layers[1]["moe"]
    assert layers[1]["ff_kind"] == B.FF_MOE and (e["experts"], e["identity"], e["top"], e["expert_ff"], e["shared_ff"]) == (5, 3, 4, 28, 0)
    assert (e["act"], e["route"], e["route_scale"], e["correction"]) == (B.ACT_SILU_GLU, B.ROUTE_SOFTMAX_TOP, 1.0, 1)
    assert layers[2]["ff"] == 0 and layers[2]["ff_kind"] == B.FF_RELU2
    assert gefovik.parse_config(cfg, 16, 1)[0]["compute"] == B.COMPUTE_BF16
    with pytest.raises(B.InvalidArgument):
        gefovik.parse_config(dict(cfg, architecture="Other"), 16, 1)
    with pytest.raises(B.Unsupported):
        gefovik.parse_config(cfg, 16, 1, "float16")
    with pytest.raises(B.Unsupported):
        gefovik.parse_config(dict(cfg, layers=[{"type": "delta", "mixer": {}}]), 16, 1)
    with pytest.raises(B.Unsupported):
        gefovik.parse_config(dict(cfg, layers=[dict(cfg["layers"][0], mlp={"kind": "other"})]), 16, 1)


def test_tensor_list_follows_the_config():
    from llama_gguf_b200 import gefovik

    cfg = S.config([S.attn(heads=6, kv_heads=2, dim=12, mlp=S.dense(12)), S.latent(heads=3, dim=16, vdim=24, kv_rank=40, mlp=S.moe(experts=3, identity=2, top=2, ff=10)),
                    S.attn(mlp=None)], width=32, vocab=50)
    t = gefovik.tensor_shapes(cfg)
    assert t["embed"] == (50, 32) and "head" not in t and t["final.norm"] == (32,)
    assert t["l0.mix.q"] == (72, 32) and t["l0.mix.k"] == (24, 32) and t["l0.mix.o"] == (32, 72) and "l0.mix.v" not in t and "l0.mix.sink" not in t
    assert t["l0.mlp.gate"] == (12, 32) and t["l0.mlp.up"] == (12, 32) and t["l0.mlp.down"] == (32, 12)
    assert t["l1.mix.q"] == (48, 32) and t["l1.mix.dkv"] == (40, 32) and t["l1.mix.dkv.norm"] == (40,) and t["l1.mix.uk"] == (48, 40)
    assert t["l1.mix.uv"] == (72, 40) and t["l1.mix.sink"] == (3,) and t["l1.mix.g"] == (3, 32) and t["l1.mix.o"] == (32, 72)
    assert t["l1.mlp.router"] == (5, 32) and t["l1.mlp.correction"] == (5,) and t["l1.mlp.e2.down"] == (32, 10) and "l1.mlp.e3.up" not in t
    assert "l2.norm2" not in t and t["l2.norm1"] == (32,)
    assert set(S.random_weights(cfg, 0)) == set(t)


def test_registry_knows_the_architecture(tmp_path):
    from llama_gguf_b200 import registry

    d = tmp_path / "model"
    d.mkdir()
    (d / "config.json").write_text(json.dumps({"architecture": "Gefovik"}))
    assert registry.architecture_of(str(d)) == "Gefovik"
    assert {"Gefovik", "Fizesun", "Marosun", "Madudra", "Mefurax", "Lazilorn"} <= set(registry.LOADERS)
