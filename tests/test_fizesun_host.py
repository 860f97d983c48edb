"""Host-side pieces of the Fizesun path that need no GPU: the oracle's pieces behave as their definitions say, config.json becomes the
right layer program, the list of tensors follows the config, the registry picks by architecture."""
import json
import math

import numpy as np
import pytest

import fizesun_oracle as O
import fizesun_synth as S


def test_norms():
    x = np.array([3.0, -4.0, 0.0, 0.0])
    assert np.allclose(O.scalar_norm(x, 2.0, 0.0), x / 2.5 * 2.0)
    assert np.allclose(O.scalar_norm(x, 2.0, 6.25), x / math.sqrt(12.5) * 2.0)          # eps inside the root
    assert np.allclose(O.weighted_norm(x, np.array([1.0, 2.0, 3.0, 4.0]), 0.0), x / 2.5 * [1, 2, 3, 4])


def test_rotation_layout():
    v = np.array([1.0, 2.0, 3.0, 4.0, 5.0])
    assert np.allclose(O.rotate_pairs(v, 0, 4, 100.0), v)
    r = O.rotate_pairs(v, 3, 4, 100.0)
    assert r[4] == 5.0
    assert abs(r[0] - (math.cos(3.0) - 2.0 * math.sin(3.0))) < 1e-12 and abs(r[1] - (2.0 * math.cos(3.0) + math.sin(3.0))) < 1e-12
    assert abs(r[2] - (3.0 * math.cos(0.3) - 4.0 * math.sin(0.3))) < 1e-12               # second pair: 100^(-2/4) = 0.1 per position
    # the score of two rotated vectors depends on the distance only
    a, b = np.random.default_rng(0).standard_normal((2, 6))
    s = [O.rotate_pairs(a, p + 5, 6, 10.0) @ O.rotate_pairs(b, p, 6, 10.0) for p in (0, 7, 100)]
    assert max(s) - min(s) < 1e-9


def test_input_convolution():
    w = np.array([[0.5, -1.0, 2.0]])
    d = O.Delay(3, 1)
    out = [O.input_convolution(np.array([h]), w, d)[0] for h in (1.0, 10.0, 100.0, 1000.0)]
    assert out == [1.0 + 2.0, 10.0 + 20.0 - 1.0, 100.0 + 200.0 - 10.0 + 0.5, 1000.0 + 2000.0 - 100.0 + 5.0]
    assert O.input_convolution(np.array([7.0]), np.array([[3.0]]), O.Delay(1, 1))[0] == 28.0


def test_xielu():
    act = np.array([0.3, -0.8])
    a, b = math.log1p(math.exp(0.3)), 0.5 + math.log1p(math.exp(-0.8))
    y = O.xielu(np.array([2.0, -1.5, 0.0]), act)
    assert abs(y[0] - (4.0 * a + 1.0)) < 1e-12 and abs(y[1] - (b * (math.exp(-1.5) + 0.5) - 0.75)) < 1e-12 and y[2] == 0.0


def test_clamped_expert():
    one = np.eye(2)
    y = O.clamped_expert(np.array([5.0, -5.0]), one, one, one, 2.0)       # gate 2 / -5, up 2 / -2
    assert abs(y[0] - 2.0 / (1.0 + math.exp(-3.404)) * 3.0) < 1e-12
    assert abs(y[1] - -5.0 / (1.0 + math.exp(8.51)) * -1.0) < 1e-12       # (the gate has no lower clamp)


def test_router_rule():
    cfg = S.config([S.latent(mlp=S.moe(experts=4, top=2, ff=3, shared_ff=5))], width=8)
    w = S.f64(S.random_weights(cfg, 1))
    h = np.random.default_rng(2).standard_normal(8)
    mlp = cfg["layers"][0]["mlp"]
    z = w["l0.mlp.router"] @ h + w["l0.mlp.router.b"]
    a, b = np.argsort(-z)[:2]
    pa = math.exp(z[a]) / (math.exp(z[a]) + math.exp(z[b]))

    def ex(name, limit):
        return O.clamped_expert(h, *(w["l0.mlp.%s.%s" % (name, k)] for k in ("gate", "up", "down")), limit)

    want = pa * ex("e%d" % a, 1.1) + (1 - pa) * ex("e%d" % b, 1.1) + ex("shared", 0.7) / (1 + math.exp(-(w["l0.mlp.shared.sg"] @ h)[0]))
    assert np.allclose(O.expert_mixture(h, w, "l0.mlp.", mlp), want)


def test_layer_runs_and_pass_entry():
    cfg = S.config([S.latent(), S.latent(), S.latent(), S.latent()], loop=(1, 3, 2))
    assert O.layer_runs(cfg) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert O.layer_runs(S.config([S.latent()])) == [(0, None)]
    W = {"loop.in": np.array([[1.0, 10.0]]), "loop.step": np.array([[0.5], [0.25]])}
    assert O.enter_pass(np.array([2.0]), np.array([3.0]), 1, W)[0] == 2.0 + 30.0 + 0.25
    # every pass keeps keys and inputs of its own
    w = S.f64(S.random_weights(cfg, 3))
    s = O.Sequence(cfg, w)
    s.token(1)
    s.token(2)
    assert [k.n for k in s.keys] == [2] * 6 and not np.allclose(s.delay[1][0].past[-1], s.delay[3][0].past[-1])


def test_parse_config_reads_every_constant():
    from llama_gguf_b200 import fizesun
    import llama_gguf_b200 as B

    cfg = S.config([S.latent(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=32, scale=0.37, base=777.0, mlp=S.moe(experts=5, top=2, ff=24, limit=1.25, shared_ff=16,
                                                                                                            shared_limit=0.75)),
                    S.latent(heads=2, mlp=S.dense(40)), S.latent()], width=64, vocab=96, eps=3e-5, taps=5, loop=(1, 3, 4))
    p, layers = fizesun.parse_config(cfg, 128, 4, "float32")
    assert (p["width"], p["vocab"], p["max_seq_len"], p["max_batch"], p["norm_eps"]) == (64, 96, 128, 4, 3e-5)
    assert (p["loop_start"], p["loop_stop"], p["loop_times"], p["loop_in"], p["in_conv"]) == (1, 3, 4, 1, 5)
    assert p["norm_scalar"] == 1 and p["embed_norm"] == 1 and p["compute"] == B.COMPUTE_F32 and p["embed_scale"] == 1.0 and p["pos_sinusoid"] == 0
    a = layers[0]["latent"]
    assert layers[0]["mixer"] == B.MIX_LATENT_ATTN
    assert (a["heads"], a["dim"], a["rot_dim"], a["vdim"], a["q_rank"], a["kv_rank"], a["mask_size"], a["kv_from"]) == (3, 16, 8, 24, 0, 32, 0, -1)
    assert a["scale"] == 0.37 and a["rot"] == {"dims": 8, "base": 777.0} and a["rot_pairs"] == 1 and a["out_gate"] == B.GATE_HEAD
    e = layers[0]["moe"]
    assert layers[0]["ff_kind"] == B.FF_MOE and (e["experts"], e["top"], e["expert_ff"], e["shared_ff"]) == (5, 2, 24, 16)
    assert (e["limit"], e["shared_limit"], e["slope"], e["router_bias"], e["shared_gate"]) == (1.25, 0.75, 1.702, 1, 1)
    assert e["act"] == B.ACT_CLAMPED_GLU and e["route"] == B.ROUTE_TOP_SOFTMAX
    assert layers[1]["ff_kind"] == B.FF_XIELU and layers[1]["ff"] == 40 and layers[1]["latent"]["heads"] == 2
    assert layers[2]["ff"] == 0 and layers[2]["ff_kind"] == B.FF_RELU2
    p2, _ = fizesun.parse_config(S.config([S.latent()]), 16, 1)
    assert p2["loop_in"] == 0 and p2["compute"] == B.COMPUTE_BF16
    with pytest.raises(B.InvalidArgument):
        fizesun.parse_config(dict(cfg, architecture="Other"), 16, 1)
    with pytest.raises(B.Unsupported):
        fizesun.parse_config(cfg, 16, 1, "float16")
    with pytest.raises(B.Unsupported):
        fizesun.parse_config(dict(cfg, layers=[{"type": "attention", "mixer": {}}]), 16, 1)


def test_tensor_list_follows_the_config():
    from llama_gguf_b200 import fizesun

    cfg = S.config([S.latent(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=40, mlp=S.moe(experts=3, top=2, ff=10, shared_ff=6)), S.latent(mlp=S.dense(12)),
                    S.latent()], width=32, vocab=50, taps=3, loop=(0, 2, 4))
    t = fizesun.tensor_shapes(cfg)
    assert t["embed"] == (50, 32) and t["embed.norm"] == () and t["loop.in"] == (32, 64) and t["loop.step"] == (4, 32)
    assert t["l0.norm1"] == () and t["l0.canon1"] == (32, 3) and t["l0.mix.q"] == (72, 32) and t["l0.mix.dkv"] == (48, 32) and t["l0.mix.dkv.norm"] == (40,)
    assert t["l0.mix.uk"] == (48, 40) and t["l0.mix.uv"] == (72, 40) and t["l0.mix.g"] == (3, 32) and t["l0.mix.o"] == (32, 72)
    assert t["l0.mlp.router"] == (3, 32) and t["l0.mlp.router.b"] == (3,) and t["l0.mlp.e2.down"] == (32, 10) and "l0.mlp.e3.up" not in t
    assert t["l0.mlp.shared.gate"] == (6, 32) and t["l0.mlp.shared.sg"] == (1, 32)
    assert t["l1.mlp.up"] == (12, 32) and t["l1.mlp.act"] == (2,) and "l1.mlp.gate" not in t
    assert "l2.norm2" not in t and "l2.canon2" not in t
    assert "loop.in" not in fizesun.tensor_shapes(S.config([S.latent()]))
    assert set(S.random_weights(cfg, 0)) == set(t)


def test_registry_knows_the_architecture(tmp_path):
    from llama_gguf_b200 import registry

    d = tmp_path / "model"
    d.mkdir()
    (d / "config.json").write_text(json.dumps({"architecture": "Fizesun"}))
    assert registry.architecture_of(str(d)) == "Fizesun"
    assert {"Fizesun", "Marosun", "Madudra", "Mefurax", "Lazilorn"} <= set(registry.LOADERS)
