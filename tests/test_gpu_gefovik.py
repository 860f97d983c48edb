"""Gefovik on the GPU against the plain oracle (tests/gefovik_oracle.py): every mechanism alone, prompts against token-by-token decoding,
portions, unequal batches, slot reuse, far keys, the steps of the query temperature, odd sizes, greedy generation through the scheduler.

The library runs in its f32 compute mode where the comparison has to be sharp (errors ~1e-6) and in bf16 mode with a bound that a
wrong mechanism exceeds by orders of magnitude."""
import copy

import numpy as np
import pytest

import gefovik_oracle as O
import gefovik_synth as S

pytestmark = pytest.mark.gpu

F32_TOL = 2e-4
BF16_TOL = 8e-2


def tokens(n, vocab, seed=1):
    return [int(t) for t in np.random.default_rng(seed).integers(0, vocab, n)]


def check_whole(cfg, n, seed=0, tol=F32_TOL, w=None):
    """f32: logits and the residual stream after every layer of one prompt, then the last third once more decoded token by token"""
    w = w if w is not None else S.random_weights(cfg, seed)
    toks = tokens(n, cfg["vocab"], seed + 1)
    want, rt = O.run(cfg, S.f64(w), toks)
    gpu = S.gpu_model(cfg, w, max_seq_len=n + 8, taps=True)
    try:
        got = gpu.step([(0, toks)], list(range(n)))
        gt = gpu.taps(n)
        assert gt.shape[0] == len(rt)
        for r in range(len(rt)):
            assert np.abs(gt[r] - rt[r]).max() <= tol * np.abs(rt[r]).max() * 4, f"residual stream after layer {r}"
        assert S.rel_err(got, want) < tol
    finally:
        gpu.close()
    gpu = S.gpu_model(cfg, w, max_seq_len=n + 8)
    try:
        cut = n - n // 3
        gpu.step([(0, toks[:cut])])
        assert S.rel_err(decoded(gpu, toks[cut:]), want[cut:]) < tol
    finally:
        gpu.close()
    return want


class Ref:
    """The oracle fed in pieces: one Sequence per request."""

    def __init__(self, cfg, w):
        self.cfg, self.w = cfg, S.f64(w)

    def new(self):
        return O.Sequence(self.cfg, self.w)

    def step(self, seq, toks):
        return np.array([seq.token(t)[0] for t in toks])

    def forward(self, toks):
        return self.step(self.new(), toks)


def decoded(gpu, toks, seq=0):
    return np.stack([gpu.forward(t, seq=seq) for t in toks])


def shows(cfg, w, toks, want, factor=50):
    """the oracle itself tells the changed model from the wanted answers"""
    return S.rel_err(Ref(cfg, w).forward(toks)[-1], want[-1]) > factor * F32_TOL


# ---------------------------------------------------------------------------------------------------- mechanisms alone
def test_attention_alone(b200):
    check_whole(S.config([S.attn()]), 40, 1)


def test_values_are_the_unnormed_keys(b200, monkeypatch):
    # keys of very different lengths: a value taken after the norm would weigh them all alike
    cfg = S.config([S.attn(heads=2, kv_heads=1)])
    w = S.random_weights(cfg, 2)
    w["embed"] = w["embed"] * np.linspace(0.2, 3.0, cfg["vocab"], dtype=np.float32)[:, None]
    want = check_whole(cfg, 30, 2, w=w)
    real = O.Rows.append
    monkeypatch.setattr(O.Rows, "append", lambda self, k, v: real(self, k=k, v=k))
    assert shows(cfg, w, tokens(30, cfg["vocab"], 3), want)


@pytest.mark.parametrize("every,coef", [(1, 0.5), (3, 0.3), (16, -0.4), (33, 1.5), (1000, 2.0)])
def test_query_temperature(b200, every, coef):
    # the factor changes where (p + 1) / every passes a whole number; the neighbouring spans and no temperature at all are told apart
    cfg = S.config([S.attn(every=every, coef=coef, scale=1.1, softcap=40.0)])
    w = S.random_weights(cfg, 4)
    n = 3 * every + 2 if every < 20 else 68
    want = check_whole(cfg, n, 4, w=w)
    toks = tokens(n, cfg["vocab"], 5)
    if every < 1000:
        steps = [p for p in range(n) if (p + 1) % every == 0]
        for other in ({"coef": 0.0, "every": every}, {"coef": coef, "every": every + 1}):
            alt = copy.deepcopy(cfg)
            alt["layers"][0]["mixer"]["q_temp"] = other
            got = Ref(alt, w).forward(toks)
            assert max(S.rel_err(got[p], want[p]) for p in steps) > 20 * F32_TOL


def test_soft_cap_bites(b200):
    cfg = S.config([S.attn(scale=2.0, softcap=2.5)])
    w = S.random_weights(cfg, 6)
    want = check_whole(cfg, 30, 6, w=w)
    for c in (2.6, 1000.0):
        alt = copy.deepcopy(cfg)
        alt["layers"][0]["mixer"]["softcap"] = c
        assert shows(alt, w, tokens(30, cfg["vocab"], 7), want, 5)


def test_latent_attention_alone(b200):
    check_whole(S.config([S.latent()]), 40, 8)


def test_sink_and_gate_matter(b200):
    cfg = S.config([S.latent(heads=2)])
    w = S.random_weights(cfg, 9)
    w["l0.mix.sink"] = np.array([4.0, -3.0], dtype=np.float32)
    want = check_whole(cfg, 30, 9, w=w)
    for name, v in (("l0.mix.sink", np.array([-30.0, -30.0])), ("l0.mix.sink", np.array([-3.0, 4.0])), ("l0.mix.g", 0 * w["l0.mix.g"])):
        assert shows(cfg, dict(w, **{name: v}), tokens(30, cfg["vocab"], 10), want)


def test_layer_norm_on_the_output(b200):
    # an epsilon of the size of the variance, an output with a large mean
    cfg = S.config([S.attn(mlp=S.dense())], eps=0.3)
    w = S.random_weights(cfg, 11)
    w["l0.mix.o"] = w["l0.mix.o"] + np.float32(0.25)
    w["l0.mlp.down"] = w["l0.mlp.down"] - np.float32(0.125)
    check_whole(cfg, 25, 11, w=w)


def test_embedding_scale_is_not_the_heads(b200):
    for scale in (1.0, 0.25, 20.0):
        check_whole(S.config([S.latent(mlp=S.dense(24))], scale=scale), 20, 12)


def test_dense_layer(b200):
    check_whole(S.config([S.attn(mlp=S.dense(72)), S.latent(mlp=S.dense(9))]), 25, 13)


def test_mixture_of_experts(b200):
    check_whole(S.config([S.attn(mlp=S.moe())]), 30, 14)
    check_whole(S.config([S.attn(mlp=S.moe(experts=3, identity=0, top=1, ff=40))]), 30, 15)             # no identity expert, one choice
    check_whole(S.config([S.attn(mlp=S.moe(experts=4, identity=3, top=7, ff=8))]), 30, 16)              # everything chosen
    check_whole(S.config([S.latent(mlp=S.moe(experts=2, identity=5, top=4, ff=16))]), 30, 17)           # more choices than experts with tensors
    check_whole(S.config([S.latent(mlp=S.moe(experts=1, identity=1, top=1, ff=12))]), 30, 18)


def test_correction_chooses_but_does_not_weigh(b200):
    cfg = S.config([S.attn(mlp=S.moe(experts=6, identity=2, top=2))])
    w = S.random_weights(cfg, 19)
    w["l0.mlp.correction"] = np.array([0, 2, 0, -2, 1.5, 0, 1.75, 0], dtype=np.float32)      # two experts, an identity one: two of them always
    want = check_whole(cfg, 30, 19, w=w)
    toks = tokens(30, cfg["vocab"], 20)
    assert shows(cfg, dict(w, **{"l0.mlp.correction": np.zeros(8)}), toks, want)


def test_identity_experts_only(b200):
    # every choice falls on identity experts: the feed-forward gives its input back, times the weights
    cfg = S.config([S.attn(mlp=S.moe(experts=4, identity=3, top=2)), S.latent()])
    w = S.random_weights(cfg, 21)
    w["l0.mlp.correction"] = np.array([-3, -3, -3, -3, 0, 0, 0], dtype=np.float32)
    check_whole(cfg, 30, 21, w=w)


def full_cfg():
    return S.config([S.attn(mlp=S.dense()), S.latent(mlp=S.moe()), S.attn(heads=3, kv_heads=3, dim=32, scale=0.2, softcap=5.0, coef=0.6, every=11, mlp=S.moe(4, 2, 3, 16)),
                     S.latent(heads=2, dim=24, vdim=20, kv_rank=48, mlp=None), S.attn(heads=6, kv_heads=1, dim=8, mlp=None), S.latent(heads=5, dim=8, vdim=16, mlp=S.dense(56))])


def test_whole_model(b200):
    check_whole(full_cfg(), 48, 22)


def near(got, want, compute, clear=True):
    """every row within the mode's bound; clear = False (bf16): rounding may have turned close calls of a router at a few positions"""
    got, want = np.atleast_2d(got), np.atleast_2d(want)
    e = np.array([S.rel_err(g, x) for g, x in zip(got, want)])
    if compute == "float32":
        return e.max() < F32_TOL
    return np.median(e) < BF16_TOL / 2 and (e < BF16_TOL).mean() >= (1.0 if clear else 0.85)


def test_bf16_mode_whole_model(b200):
    cfg = full_cfg()
    toks = tokens(48, cfg["vocab"], 23)
    w = S.clear_weights(cfg, [toks], 22)
    want = Ref(cfg, w).forward(toks)
    gpu = S.gpu_model(cfg, w, "bfloat16")
    try:
        assert near(gpu.step([(0, toks)], list(range(48))), want, "bfloat16")
    finally:
        gpu.close()


@pytest.mark.parametrize("layers,width", [
    ([S.attn(heads=1, kv_heads=1, dim=10, mlp=S.dense(9)), S.latent(heads=1, dim=10, vdim=7, kv_rank=18)], 40),                 # sizes no vector load takes
    ([S.attn(heads=3, kv_heads=1, dim=7, mlp=S.moe(3, 1, 2, 5)), S.latent(heads=5, dim=3, vdim=5, kv_rank=17, mlp=S.moe(2, 2, 3, 7))], 37),   # odd everywhere
    ([S.attn(heads=2, kv_heads=1, dim=80, mlp=S.moe(2, 1, 1, 4)), S.latent(heads=2, dim=40, vdim=72, kv_rank=136, mlp=S.dense(12))], 72),
    ([S.attn(heads=12, kv_heads=1, dim=16, mlp=S.dense(136)), S.latent(heads=9, dim=16, vdim=8, kv_rank=64)], 48),               # heads beyond one group of eight
    ([S.attn(heads=20, kv_heads=2, dim=12), S.latent(heads=17, dim=8, vdim=16, kv_rank=24)], 32),
    ([S.attn(heads=2, kv_heads=2, dim=144, scale=0.05), S.attn(heads=2, kv_heads=1, dim=272, scale=0.04, mlp=S.dense(8))], 64),    # wide heads
    ([S.latent(heads=2, dim=16, vdim=24, kv_rank=300, mlp=S.moe(9, 3, 4, 12)), S.attn(heads=8, kv_heads=4, dim=4)], 56),           # wide latent
])
@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_other_sizes(b200, layers, width, compute):
    cfg = S.config(layers, width=width, vocab=50, eps=3e-4)
    toks = tokens(33, cfg["vocab"], 25)
    w = S.clear_weights(cfg, [toks], 24)
    want = Ref(cfg, w).forward(toks)
    gpu = S.gpu_model(cfg, w, compute)
    try:
        assert near(gpu.step([(0, toks[:26])], list(range(26))), want[:26], compute)
        assert near(decoded(gpu, toks[26:]), want[26:], compute)
    finally:
        gpu.close()


# ---------------------------------------------------------------------------------------------------- prompts, portions, batches
def test_prompt_against_token_by_token(b200):
    cfg = full_cfg()
    w = S.random_weights(cfg, 26)
    toks = tokens(34, cfg["vocab"], 27)
    want = Ref(cfg, w).forward(toks)
    gpu = S.gpu_model(cfg, w)
    try:
        assert S.rel_err(decoded(gpu, toks), want) < F32_TOL        # every token decoded alone, from the first one
        assert gpu.position() == len(toks)
        gpu.reset()
        last = gpu.forward_batch(toks[:20])                         # prompt, then decoding
        assert S.rel_err(last, want[19]) < F32_TOL
        assert S.rel_err(decoded(gpu, toks[20:]), want[20:]) < F32_TOL
    finally:
        gpu.close()


@pytest.mark.parametrize("portion", [2, 3, 7, 16, 17])
def test_portions(b200, portion):
    cfg = full_cfg()
    toks = tokens(37, cfg["vocab"], 29)
    w = S.clear_weights(cfg, [toks], 28)
    want = Ref(cfg, w).forward(toks)
    for compute in ("float32", "bfloat16"):
        gpu = S.gpu_model(cfg, w, compute)
        try:
            got = []
            for a in range(0, len(toks), portion):
                part = toks[a:a + portion]
                got.append(gpu.step([(1, part)], list(range(len(part)))))
            assert near(np.concatenate(got), want, compute)
        finally:
            gpu.close()


def test_portions_between_decoded_tokens(b200):
    # prompts, single tokens and short portions in turn: the decoding kernels and the prompt kernels share one cache
    cfg = full_cfg()
    cuts = [1, 1, 2, 1, 5, 1, 1, 1, 3, 9, 1, 2, 2, 12, 1]
    toks = tokens(sum(cuts), cfg["vocab"], 31)
    w = S.clear_weights(cfg, [toks], 30)
    want = Ref(cfg, w).forward(toks)
    for compute in ("float32", "bfloat16"):
        gpu = S.gpu_model(cfg, w, compute)
        try:
            got, a = [], 0
            for n in cuts:
                got.append(gpu.step([(2, toks[a:a + n])], list(range(n))))
                a += n
            assert near(np.concatenate(got), want, compute)
        finally:
            gpu.close()


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_unequal_batch_against_each_alone(b200, compute):
    cfg = full_cfg()
    prompts = [tokens(n, cfg["vocab"], 20 + n) for n in (1, 9, 18, 5)]
    tails = [tokens(9, cfg["vocab"], 40 + i) for i in range(4)]
    w = S.clear_weights(cfg, [p + t[:3 + 2 * i] for i, (p, t) in enumerate(zip(prompts, tails))], 32, margin=0.01)
    ref = Ref(cfg, w)
    gpu = S.gpu_model(cfg, w, compute, max_batch=6)
    try:
        slots = [4, 0, 2, 5]
        got = gpu.step(list(zip(slots, prompts)), list(range(sum(len(p) for p in prompts))))
        states = [ref.new() for _ in prompts]
        assert near(got, np.concatenate([ref.step(st, p) for st, p in zip(states, prompts)]), compute)
        rows, want = [], []
        for k in range(9):                                          # the shortest request ends first, then the next one
            alive = [i for i in range(4) if k < 3 + 2 * i]
            lg = gpu.decode_batch([slots[i] for i in alive], [tails[i][k] for i in alive])
            for j, i in enumerate(alive):
                rows.append(lg[j])
                want.append(ref.step(states[i], [tails[i][k]])[0])
        assert near(np.array(rows), np.array(want), compute)
    finally:
        gpu.close()


def test_mixed_batch_of_prompts_and_single_tokens(b200):
    cfg = full_cfg()
    w = S.random_weights(cfg, 33)
    ref = Ref(cfg, w)
    a, b, c = (tokens(n, cfg["vocab"], 60 + n) for n in (21, 18, 30))
    gpu = S.gpu_model(cfg, w)
    try:
        gpu.step([(0, a[:11])])
        got = gpu.step([(1, b[:17]), (0, a[11:12]), (3, c[:2])], list(range(20)))      # a new prompt, one decoded token, a short prompt
        wa, wb, wc = ref.forward(a), ref.forward(b), ref.forward(c)
        assert S.rel_err(got, np.concatenate([wb[:17], wa[11:12], wc[:2]])) < F32_TOL
        got = gpu.step([(0, a[12:]), (3, c[2:]), (1, b[17:])], list(range(9 + 28 + 1)))
        assert S.rel_err(got, np.concatenate([wa[12:], wc[2:], wb[17:]])) < F32_TOL
    finally:
        gpu.close()


@pytest.mark.parametrize("rows", [2, 3, 5, 8, 11, 16, 24, 40, 70])
def test_decoding_many_sequences(b200, rows):
    # every row count the few-row kernels are built for, and the counts beyond them
    cfg = S.config([S.attn(heads=6, kv_heads=2, mlp=S.moe(5, 2, 2, 24)), S.latent(heads=10, mlp=S.dense()), S.attn(heads=2, kv_heads=2, dim=32, mlp=S.dense(64))])
    w = S.random_weights(cfg, 34)
    ref = Ref(cfg, w)
    seqs = [tokens(3 + (5 * i) % 7, cfg["vocab"], 100 + i) for i in range(rows)]
    tails = [tokens(3, cfg["vocab"], 200 + i) for i in range(rows)]
    want = np.concatenate([ref.forward(seqs[i] + tails[i])[len(seqs[i]):] for i in range(rows)])
    for compute in ("float32", "bfloat16"):
        gpu = S.gpu_model(cfg, w, compute, max_batch=rows, max_seq_len=32)
        try:
            gpu.step([(i, t) for i, t in enumerate(seqs)])
            got = np.stack([gpu.decode_batch(list(range(rows)), [t[k] for t in tails]) for k in range(3)], axis=1)
            assert near(got.reshape(3 * rows, -1), want, compute, clear=False)
        finally:
            gpu.close()


def test_slots_freed_and_used_again(b200):
    cfg = full_cfg()
    w = S.random_weights(cfg, 35)
    ref = Ref(cfg, w)
    gpu = S.gpu_model(cfg, w, max_batch=3)
    try:
        assert gpu.pool_counts() == (0, 0)
        a, b, c = tokens(30, cfg["vocab"], 3), tokens(18, cfg["vocab"], 4), tokens(25, cfg["vocab"], 5)
        gpu.step([(0, a), (1, b)])
        assert gpu.pool_counts() == (2, 0)
        gpu.reset(0)
        assert gpu.pool_counts() == (1, 1) and gpu.position(0) == 0
        # slot 2 takes the block that slot 0 left (full of a's rows and factors); slot 1 goes on undisturbed
        got = np.concatenate([gpu.step([(2, c[:1])], [0]), gpu.step([(2, c[1:])], list(range(24)))])
        assert gpu.pool_counts() == (2, 0)
        assert S.rel_err(got, ref.forward(c)) < F32_TOL
        st = ref.new()
        ref.step(st, b)
        for t in tokens(5, cfg["vocab"], 6):
            assert S.rel_err(gpu.forward(t, seq=1), ref.step(st, [t])[0]) < F32_TOL
        gpu.reset(2)
        gpu.reset(1)
        got = gpu.step([(1, a)], [len(a) - 1])
        assert S.rel_err(got, ref.forward(a)[-1]) < F32_TOL
    finally:
        gpu.close()


# ---------------------------------------------------------------------------------------------------- far keys, edges, first tokens
def planted_key_model(kind, dim=16):
    """One layer in which the probe token's queries point at the needle token's key.  Fewer tokens than the width, and the mixer reads the
    scaled embedding row itself: a vector g with g . x = 1 for the needle's row and 0 for every other token's exists, so W + (big u) g^T
    turns the needle's key (or latent) alone into the direction u, the mean direction of the probe's queries.  Its score stands out among
    hundreds of random ones in every head."""
    mixer = S.attn(heads=4, kv_heads=2, dim=dim, scale=12.0 / dim, softcap=30.0, coef=0.1, every=50) if kind == "attention" else \
        S.latent(heads=2, dim=16, vdim=24, kv_rank=dim, scale=1.0)
    cfg = S.config([mixer], width=48, vocab=40)
    w = S.random_weights(cfg, 36)
    needle, probe = cfg["vocab"] - 2, cfg["vocab"] - 1
    W, m = S.f64(w), cfg["layers"][0]["mixer"]
    x = W["embed"] * cfg["embedding"]["scale"]
    g = np.linalg.pinv(x)[:, needle]
    assert np.abs(x @ g - np.eye(cfg["vocab"])[needle]).max() < 1e-9
    q = (W["l0.mix.q"] @ x[probe]).reshape(m["heads"], m["dim"])
    if kind == "attention":
        k = np.array(W["l0.mix.k"]).reshape(m["kv_heads"], m["dim"], -1)
        per = m["heads"] // m["kv_heads"]
        for j in range(m["kv_heads"]):
            u = (q[j * per:(j + 1) * per] / np.linalg.norm(q[j * per:(j + 1) * per], axis=1, keepdims=True)).sum(axis=0)
            k[j] += np.outer(20.0 * u / np.linalg.norm(u), g)
        w["l0.mix.k"] = k.reshape(w["l0.mix.k"].shape).astype(np.float32)
    else:
        w["l0.mix.dkv.norm"] = np.ones_like(w["l0.mix.dkv.norm"])
        w["l0.mix.g"] = 0.2 * w["l0.mix.g"]
        uk = W["l0.mix.uk"].reshape(m["heads"], m["dim"], m["kv_rank"])
        qa = np.stack([uk[h].T @ q[h] for h in range(m["heads"])])
        u = (qa / np.linalg.norm(qa, axis=1, keepdims=True)).sum(axis=0)
        w["l0.mix.dkv"] = (W["l0.mix.dkv"] + np.outer(60.0 * u / np.linalg.norm(u), g)).astype(np.float32)
    return cfg, w, needle, probe


@pytest.mark.parametrize("kind,dim", [("attention", 16), ("attention", 80), ("attention", 160), ("latent", 32), ("latent", 160)])
def test_far_key_among_hundreds(b200, kind, dim):
    # probes from position 290 on, in a prompt and decoded, meet a needle at the very start, at the borders of the kernels' key tiles and
    # in between
    cfg, w, needle, probe = planted_key_model(kind, dim)
    n, cut = 304, 297
    ref = Ref(cfg, w)
    base = tokens(n, cfg["vocab"] - 2, 37)
    base[290:] = [probe] * (n - 290)
    plain = ref.forward(base)
    for at in ((0, 1, 31, 32, 63, 64, 127, 200) if dim < 80 else (0, 31, 64)):
        toks = list(base)
        toks[at] = needle
        want = ref.forward(toks)
        assert min(S.rel_err(plain[p], want[p]) for p in (290, 296, 300)) > 40 * F32_TOL
        for compute, tol in (("float32", F32_TOL), ("bfloat16", BF16_TOL)):
            gpu = S.gpu_model(cfg, w, compute, max_seq_len=n + 4)
            try:
                got = gpu.step([(0, toks[:cut])], list(range(290, cut)))
                assert S.rel_err(got, want[290:cut]) < tol, at
                assert S.rel_err(decoded(gpu, toks[cut:]), want[cut:]) < tol, at
            finally:
                gpu.close()


def test_first_tokens_and_long_decoding(b200):
    cfg = full_cfg()
    w = S.random_weights(cfg, 38)
    toks = tokens(140, cfg["vocab"], 39)      # decoded one by one from the very first token, over several key tiles
    want = Ref(cfg, w).forward(toks)
    gpu = S.gpu_model(cfg, w)
    try:
        got = decoded(gpu, toks)
        for p in range(len(toks)):
            assert S.rel_err(got[p], want[p]) < F32_TOL, p
    finally:
        gpu.close()


def test_long_prompt_then_decoding(b200):
    # more keys than the decoding kernels' splits have tiles, positions where the temperature has stepped often
    cfg = S.config([S.attn(heads=2, kv_heads=1, every=90, coef=0.7), S.latent(heads=2)], width=32, vocab=40)
    w = S.random_weights(cfg, 40)
    n = 2230
    toks = tokens(n, cfg["vocab"], 41)
    want = Ref(cfg, w).forward(toks)
    for compute in ("float32", "bfloat16"):
        gpu = S.gpu_model(cfg, w, compute, max_seq_len=n + 4)
        try:
            assert near(gpu.step([(0, toks[:2200])], list(range(2150, 2200))), want[2150:2200], compute)
            assert near(decoded(gpu, toks[2200:]), want[2200:], compute)
        finally:
            gpu.close()


def test_row_does_not_depend_on_the_batch(b200):
    cfg = full_cfg()
    w = S.random_weights(cfg, 42)
    a, b = tokens(21, cfg["vocab"], 1), tokens(40, cfg["vocab"], 2)
    for compute, tol in (("float32", 1e-5), ("bfloat16", 3e-2)):
        gpu = S.gpu_model(cfg, w, compute)
        try:
            alone = gpu.step([(0, a)], list(range(len(a))))
            both = gpu.step([(1, b), (2, a)], list(range(len(b), len(b) + len(a))))
            assert S.rel_err(both, alone) < tol
        finally:
            gpu.close()


# ---------------------------------------------------------------------------------------------------- generation through the scheduler
def test_greedy_generation_through_the_batched_engine(b200):
    cfg = full_cfg()
    w = S.random_weights(cfg, 43)
    prompts = [tokens(n, cfg["vocab"], 50 + n) for n in (5, 17, 9, 26, 3)]
    n_new = [6, 4, 8, 5, 7]
    want = [O.greedy(cfg, S.f64(w), p, k) for p, k in zip(prompts, n_new)]
    gpu = S.gpu_model(cfg, w, max_batch=3)
    eng = b200.BatchedEngine(gpu, max_batch_size=3, max_seq_len=200, eos_token_id=cfg["vocab"] + 7)   # (no token is EOS)
    try:
        ids = [eng.submit(p, k) for p, k in zip(prompts, n_new)]   # five requests on three slots: two wait, slots are reused
        got = {i: [] for i in ids}
        done = {}
        for ev in eng.run():
            if ev[0] == "token":
                got[ev[1]].append(ev[2])
            elif ev[0] == "done":
                done[ev[1]] = ev[2:]
            else:
                raise AssertionError(ev)
        for i, rid in enumerate(ids):
            assert got[rid] == want[i], i
            assert done[rid] == ("max_tokens", len(prompts[i]), n_new[i])
        assert gpu.pool_counts()[0] <= 3
    finally:
        eng.close()
        gpu.close()


def test_decode_greedy_entry_point(b200):
    cfg = full_cfg()
    w = S.random_weights(cfg, 44)
    p = tokens(12, cfg["vocab"], 45)
    want = O.greedy(cfg, S.f64(w), p, 6)
    gpu = S.gpu_model(cfg, w)
    try:
        first = gpu.step([(0, p)], [len(p) - 1])[0]
        t0 = int(len(first) - 1 - np.argmax(first[::-1]))
        assert t0 == want[0]
        out, _ = gpu.decode_greedy(t0, 5)
        assert out.tolist() == want[1:]
    finally:
        gpu.close()


def test_bad_arguments(b200):
    from llama_gguf_b200 import gefovik

    cfg = full_cfg()
    w = S.random_weights(cfg, 46)
    short = dict(w)
    del short["l1.mlp.correction"]
    with pytest.raises(b200.InvalidArgument):
        S.gpu_model(cfg, short)
    wrong = dict(w)
    wrong["l1.mix.sink"] = np.ones(7, dtype=np.float32)
    with pytest.raises(b200.ShapeMismatch):
        S.gpu_model(cfg, wrong)
    program, layers = gefovik.parse_config(cfg, 64, 2, "float32")
    for bad in (dict(program, post_norm=3), dict(program, streams=2), dict(program, parallel_ff=1), dict(program, loop_stop=2, loop_times=2)):
        with pytest.raises(b200.InvalidArgument):
            b200.LayerProgramInference(bad, layers, {})
    for part, field, value in (("sattn", "vdim", 24), ("sattn", "qkv_bias", 1), ("sattn", "q_temp_every", -1), ("moe", "top", 99), ("moe", "identity", -1)):
        bad = copy.deepcopy(layers)
        bad[2][part][field] = value
        with pytest.raises(b200.InvalidArgument):
            b200.LayerProgramInference(program, bad, {})


# ---------------------------------------------------------------------------------------------------- kernels against their plain forms
@pytest.mark.parametrize("layer", [S.attn(heads=8, kv_heads=2, dim=64), S.attn(heads=5, kv_heads=1, dim=16), S.attn(heads=4, kv_heads=4, dim=128, scale=0.1),
                                   S.attn(heads=2, kv_heads=1, dim=24), S.attn(heads=14, kv_heads=2, dim=48), S.attn(heads=2, kv_heads=1, dim=176, scale=0.1),
                                   S.latent(heads=3, kv_rank=64), S.latent(heads=1, kv_rank=96), S.latent(heads=7, kv_rank=224)])
def test_tile_attention_against_warp_attention(b200, monkeypatch, layer):
    # bf16 prompts of 16 rows and more take the tensor-pipe tile kernel when the cached row is a multiple of 16 wide (fourth case: it is not);
    # B200_LP_ATTN_TILE=0 keeps the warp kernel
    cfg = S.config([layer], width=64, vocab=64)
    w = S.random_weights(cfg, 47)
    a, b = tokens(190, cfg["vocab"], 48), tokens(70, cfg["vocab"], 49)
    want = Ref(cfg, w).forward(a)
    out = {}
    for tile in ("1", "0"):
        monkeypatch.setenv("B200_LP_ATTN_TILE", tile)
        gpu = S.gpu_model(cfg, w, "bfloat16")
        try:
            gpu.step([(0, a[:37])])
            out[tile] = gpu.step([(1, b), (0, a[37:])], list(range(len(b), len(b) + len(a) - 37)))
        finally:
            gpu.close()
    d = np.array([S.rel_err(x, y) for x, y in zip(out["1"], out["0"])])
    assert S.rel_err(out["1"], want[37:]) < BF16_TOL
    assert np.median(d) < 1e-2 and d.max() < BF16_TOL / 2


def test_tensor_core_gemm_path(b200, monkeypatch):
    # bf16 steps of 17 rows and more multiply on the tensor cores, the gated products and the experts' grouped products included
    cfg = full_cfg()
    w = S.random_weights(cfg, 50)
    toks = tokens(200, cfg["vocab"], 51)
    want = Ref(cfg, w).forward(toks)
    out = {}
    for tc in ("1", "0"):
        monkeypatch.setenv("B200_LP_TC", tc)
        gpu = S.gpu_model(cfg, w, "bfloat16")
        try:
            out[tc] = gpu.step([(0, toks)], list(range(len(toks))))
        finally:
            gpu.close()
    d = np.array([S.rel_err(out["1"][i], out["0"][i]) for i in range(len(toks))])
    assert np.median(d) < 2e-2 and (d < 4e-2).mean() > 0.9
    assert near(out["1"], want, "bfloat16", clear=False)


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
@pytest.mark.parametrize("env", [{}, {"B200_LP_FUSE": "0"}, {"B200_LP_LAT_SPLIT": "0"}, {"B200_LP_GRAPH": "0"}, {"B200_LP_FUSE": "0", "B200_LP_GRAPH": "0"}])
@pytest.mark.parametrize("n", [1, 2, 3])
def test_decode_kernels_against_the_unfused_forms(b200, monkeypatch, env, compute, n):
    cfg = full_cfg()
    prompts = [tokens(k, cfg["vocab"], 60 + k) for k in (3, 11, 1)[:n]]
    tails = [tokens(8, cfg["vocab"], 70 + i) for i in range(n)]
    w = S.clear_weights(cfg, [p + t for p, t in zip(prompts, tails)], 52)
    ref = Ref(cfg, w)
    states = [ref.new() for _ in prompts]
    for st, pr in zip(states, prompts):
        ref.step(st, pr)
    want = np.array([[ref.step(states[i], [tails[i][k]])[0] for i in range(n)] for k in range(8)])
    for k, v in env.items():
        monkeypatch.setenv(k, v)
    gpu = S.gpu_model(cfg, w, compute)
    try:
        gpu.step([(i, pr) for i, pr in enumerate(prompts)])
        got = np.array([gpu.decode_batch(list(range(n)), [tails[i][k] for i in range(n)]) for k in range(8)])
        assert near(got.reshape(8 * n, -1), want.reshape(8 * n, -1), compute)
    finally:
        gpu.close()


@pytest.mark.parametrize("rows", [3, 7, 9, 16])
def test_small_batches_on_the_tensor_pipe(b200, monkeypatch, rows):
    # bf16 steps of 3 to 16 rows: products with K a multiple of 32 run on mma.sync (here every one; output counts that no tile of 16 divides
    # included), and rows that choose more experts than there are take every expert once; B200_LP_GEMV_MMA=0 keeps the CUDA-core kernels
    cfg = S.config([S.attn(heads=6, kv_heads=2, mlp=S.moe(4, 2, 2, 32)), S.latent(heads=4, vdim=16, mlp=S.dense(96))], width=96, vocab=101)
    w = S.random_weights(cfg, 53)
    ref = Ref(cfg, w)
    prompts = [tokens(2 + i % 5, cfg["vocab"], 80 + i) for i in range(rows)]
    tails = [tokens(4, cfg["vocab"], 120 + i) for i in range(rows)]
    out = {}
    for mma in ("1", "0"):
        monkeypatch.setenv("B200_LP_GEMV_MMA", mma)
        gpu = S.gpu_model(cfg, w, "bfloat16", max_batch=rows, max_seq_len=32)
        try:
            gpu.step(list(enumerate(prompts)))
            out[mma] = np.stack([gpu.decode_batch(list(range(rows)), [t[k] for t in tails]) for k in range(4)])
        finally:
            gpu.close()
    d = np.array([[S.rel_err(out["1"][k][i], out["0"][k][i]) for i in range(rows)] for k in range(4)])
    assert np.median(d) < 2e-2 and (d < 4e-2).mean() > 0.85
    want = [ref.forward(prompts[i] + tails[i])[len(prompts[i]):] for i in range(rows)]
    e = np.array([[S.rel_err(out["1"][k][i], want[i][k]) for i in range(rows)] for k in range(4)])
    assert np.median(e) < BF16_TOL / 2


# ---------------------------------------------------------------------------------------------------- the mechanisms in other layer forms
def test_options_in_other_layer_forms(b200):
    """The query temperature without v_from_k, the sink of latent attention, identity experts and the corrected choice in the norm-first form
    and in the norm-after-sum form, an untied head: each against the same program in its other kernels (prompt, few rows, single tokens)."""
    sattn = {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 8, "mask": b200.MASK_CAUSAL, "scale": 0.3, "softcap": 6.0, "qk_norm": b200.QKNORM_HEAD_UNIT,
             "q_temp_coef": 0.5, "q_temp_every": 5}
    lat = {"heads": 3, "dim": 8, "vdim": 8, "kv_rank": 16, "scale": 0.35, "kv_from": -1, "out_gate": b200.GATE_HEAD, "sink": b200.SINK_LEARNED}
    e = {"experts": 4, "identity": 2, "top": 3, "expert_ff": 16, "act": b200.ACT_SILU_GLU, "route": b200.ROUTE_SIGMOID_TOP, "correction": 1}
    W, V = 32, 48
    rng = np.random.default_rng(54)
    shapes = {"embed": (V, W), "head": (V, W), "final.norm": (W,), "l0.norm1": (W,), "l0.norm2": (W,), "l1.norm1": (W,), "l1.norm2": (W,),
              "l0.mix.q": (64, W), "l0.mix.k": (32, W), "l0.mix.v": (16, W), "l0.mix.o": (W, 32), "l1.mix.q": (24, W), "l1.mix.dkv": (16, W),
              "l1.mix.dkv.norm": (16,), "l1.mix.uk": (24, 16), "l1.mix.uv": (24, 16), "l1.mix.g": (3, W), "l1.mix.sink": (3,), "l1.mix.o": (W, 24),
              "l1.mlp.gate": (40, W), "l1.mlp.up": (40, W), "l1.mlp.down": (W, 40), "l0.mlp.router": (6, W), "l0.mlp.correction": (6,)}
    for j in range(4):
        shapes.update({"l0.mlp.e%d.gate" % j: (16, W), "l0.mlp.e%d.up" % j: (16, W), "l0.mlp.e%d.down" % j: (W, 16)})
    tensors = {n: (b200.F32, list(reversed(s)), (rng.standard_normal(s) * (0.5 if len(s) == 1 else s[-1] ** -0.5) + (1.0 if "norm" in n else 0.0)).astype(np.float32))
               for n, s in shapes.items()}
    toks = tokens(41, V, 55)
    layers = [{"mixer": b200.MIX_SOFTMAX_ATTN, "sattn": sattn, "ff_kind": b200.FF_MOE, "moe": e},
              {"mixer": b200.MIX_LATENT_ATTN, "latent": lat, "ff": 40, "ff_kind": b200.FF_GATED_RELU}]
    seen = []
    for form in (b200.FORM_NORM_FIRST, b200.FORM_NORM_SUM):
        program = {"width": W, "vocab": V, "max_seq_len": 64, "max_batch": 4, "norm_eps": 1e-5, "embed_scale": 2.0, "logit_scale": 1.0,
                   "compute": b200.COMPUTE_F32, "post_norm": form, "residual_alpha": 1.0}
        gpu = b200.LayerProgramInference(program, layers, tensors)
        try:
            whole = gpu.step([(0, toks)], list(range(41)))
            parts = np.concatenate([gpu.step([(1, toks[:3])], [0, 1, 2]), gpu.step([(1, toks[3:12])], list(range(9))), decoded(gpu, toks[12:20], 1),
                                    gpu.step([(1, toks[20:])], list(range(21)))])
            assert np.isfinite(whole).all() and S.rel_err(parts, whole) < F32_TOL
            pair = gpu.step([(2, toks[:9]), (3, toks[:7])], list(range(16)))
            assert S.rel_err(pair, np.concatenate([whole[:9], whole[:7]])) < F32_TOL
        finally:
            gpu.close()
        seen.append(whole)
        # every option shows
        for part, field, value in (("sattn", "q_temp_every", 0), ("latent", "sink", b200.SINK_NONE), ("moe", "correction", 0)):
            alt = copy.deepcopy(layers)
            alt[0 if part != "latent" else 1][part][field] = value
            gpu = b200.LayerProgramInference(program, alt, tensors)
            try:
                assert S.rel_err(gpu.step([(0, toks)], list(range(41))), whole) > 20 * F32_TOL, field
            finally:
                gpu.close()
    assert S.rel_err(seen[0], seen[1]) > 20 * F32_TOL


def test_trace_runner_on_a_model_folder(b200, tmp_path):
    # config.json + model.safetensors (bf16) on disk -> registry -> bin/trace_run: two requests start together with unequal prompts, are
    # decoded together, the shorter one ends first; logits of the wanted rows come back in files
    import json
    import os
    import subprocess
    import sys

    from llama_gguf_b200.safetensors_io import bf16_bits, write_safetensors

    cfg = full_cfg()
    w = S.random_weights(cfg, 56)
    d = tmp_path / "model"
    d.mkdir()
    (d / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(d / "model.safetensors"), {n: bf16_bits(a).reshape(a.shape) for n, a in w.items()})
    a, b = tokens(19, cfg["vocab"], 57), tokens(7, cfg["vocab"], 58)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:15], "want": [0, 14]}, {"id": "y", "tokens": b[:5], "want": [4]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[15:16], "want": []}, {"id": "y", "tokens": b[5:6], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": a[16:17], "want": [0]}, {"id": "y", "tokens": b[6:7], "want": [0]}], "end": ["y"]},
             {"step": 3, "entries": [{"id": "x", "tokens": a[17:19], "want": [1]}], "end": ["x"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(d), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.split("\n") if ln.startswith("done")] == ["done %d" % i for i in range(4)]
    ref = Ref(cfg, w)
    wa, wb = ref.forward(a), ref.forward(b)
    got = {i: np.fromfile(str(out / ("%d.f32" % i)), dtype="<f4").reshape(-1, cfg["vocab"]) for i in range(4)}
    assert S.rel_err(got[0], np.stack([wa[0], wa[14], wb[4]])) < F32_TOL
    assert S.rel_err(got[1], wb[5:6]) < F32_TOL
    assert S.rel_err(got[2], np.stack([wa[16], wb[6]])) < F32_TOL
    assert S.rel_err(got[3], wa[18:19]) < F32_TOL
