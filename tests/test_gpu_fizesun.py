"""Fizesun on the GPU against the plain oracle (tests/fizesun_oracle.py): every mechanism alone, prompts against token-by-token decoding,
portions, unequal batches, slot reuse, the edges of the input convolution, far keys, repeated ranges, odd sizes, greedy generation
through the scheduler.

The library runs in its f32 compute mode where the comparison has to be sharp (errors ~1e-6) and in bf16 mode with a bound that a
wrong mechanism exceeds by orders of magnitude."""
import copy

import numpy as np
import pytest

import fizesun_oracle as O
import fizesun_synth as S

pytestmark = pytest.mark.gpu

F32_TOL = 2e-4
BF16_TOL = 8e-2


def tokens(n, vocab, seed=1):
    return [int(t) for t in np.random.default_rng(seed).integers(0, vocab, n)]


def check_whole(cfg, n, seed=0, compute="float32", tol=F32_TOL, taps=True, w=None):
    w = w if w is not None else S.random_weights(cfg, seed)
    toks = tokens(n, cfg["vocab"], seed + 1)
    want, rt = O.run(cfg, S.f64(w), toks)
    gpu = S.gpu_model(cfg, w, compute, max_seq_len=n + 8, taps=taps)
    try:
        got = gpu.step([(0, toks)], list(range(n)))
        if taps:
            gt = gpu.taps(n)
            assert gt.shape[0] == len(rt)
            for r in range(len(rt)):
                assert np.abs(gt[r] - rt[r]).max() <= tol * np.abs(rt[r]).max() * 4, f"residual stream after layer run {r}"
        assert S.rel_err(got, want) < tol
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


# ---------------------------------------------------------------------------------------------------- mechanisms alone
def test_latent_attention_alone(b200):
    check_whole(S.config([S.latent()], taps=1), 40, 1)


def test_embedding_norm_and_one_number_norms(b200):
    # gains far from 1 and of both signs; a weight per coordinate or a norm left out would move everything
    cfg = S.config([S.latent(mlp=S.dense())], taps=1)
    w = S.random_weights(cfg, 2)
    for name, v in (("embed.norm", 2.5), ("l0.norm1", -1.5), ("l0.norm2", 0.25), ("final.norm", 3.0)):
        w[name] = np.float32(v).reshape(())
    check_whole(cfg, 20, 2, w=w)


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 7])
def test_input_convolution(b200, taps):
    check_whole(S.config([S.latent(mlp=S.dense()), S.latent()], taps=taps), 30, 3)


def test_dense_xielu(b200):
    # both numbers of the activation away from each other and from zero
    cfg = S.config([S.latent(mlp=S.dense(72))], taps=2)
    w = S.random_weights(cfg, 4)
    for act in ((-1.5, 2.0), (1.25, -0.75)):
        w["l0.mlp.act"] = np.array(act, dtype=np.float32)
        check_whole(cfg, 25, 4, w=w)


def test_mixture_of_experts(b200):
    check_whole(S.config([S.latent(mlp=S.moe())], taps=2), 30, 5)
    check_whole(S.config([S.latent(mlp=S.moe(experts=7, top=7, ff=8, shared_ff=40))], taps=2), 30, 6)        # every expert chosen
    check_whole(S.config([S.latent(mlp=S.moe(experts=3, top=1, ff=40, limit=0.4, shared_ff=8, shared_limit=2.5))], taps=2), 30, 7)
    check_whole(S.config([S.latent(mlp=S.moe(shared_ff=0))], taps=2), 30, 8)                                 # no shared expert


def test_router_bias_decides(b200):
    # a bias that turns the choice of most tokens around
    cfg = S.config([S.latent(mlp=S.moe(experts=6, top=2))], taps=2)
    w = S.random_weights(cfg, 9)
    w["l0.mlp.router"] = 0.3 * w["l0.mlp.router"]
    w["l0.mlp.router.b"] = np.array([0, 3, 0, -3, 5, 0], dtype=np.float32)
    want = check_whole(cfg, 30, 9, w=w)
    w2 = dict(w)
    w2["l0.mlp.router.b"] = np.zeros(6, dtype=np.float32)
    assert S.rel_err(Ref(cfg, w2).forward(tokens(30, cfg["vocab"], 10)), want) > 100 * F32_TOL


def test_clamps_are_hit(b200):
    # expert inputs far beyond the limits on both sides; the limits of experts and shared expert differ
    cfg = S.config([S.latent(mlp=S.moe(limit=0.5, shared_limit=1.75))], taps=2)
    w = S.random_weights(cfg, 10)
    for k in w:
        if ".mlp." in k and (k.endswith(".gate") or k.endswith(".up")):
            w[k] = 4.0 * w[k]
    want = check_whole(cfg, 30, 10, w=w)
    for which in ("expert", "shared"):
        alt = copy.deepcopy(cfg)
        alt["layers"][0]["mlp"][which]["limit"] *= 1.2
        assert S.rel_err(Ref(alt, w).forward(tokens(30, cfg["vocab"], 11)), want) > 20 * F32_TOL


@pytest.mark.parametrize("loop", [(0, 2, 3), (1, 2, 2), (1, 3, 1), (0, 3, 2)])
def test_repeated_range(b200, loop):
    cfg = S.config([S.latent(mlp=S.dense()), S.latent(heads=2, mlp=S.moe()), S.latent(mlp=S.dense(24))], taps=3, loop=loop)
    check_whole(cfg, 24, 11)


def full_cfg():
    return S.config([S.latent(mlp=S.moe()), S.latent(heads=2, dim=24, rot_dim=16, vdim=20, kv_rank=48, base=333.0, mlp=S.dense()),
                     S.latent(heads=4, dim=8, vdim=16, mlp=S.moe(experts=4, top=3, ff=16, limit=2.0, shared_ff=24)), S.latent(mlp=None)],
                    taps=4, loop=(1, 3, 2))


def test_whole_model(b200):
    check_whole(full_cfg(), 48, 12)


def test_bf16_mode_whole_model(b200):
    # row by row: rounding may turn a close call of a router at a single position, so the bound holds for nearly all rows
    cfg = full_cfg()
    w = S.random_weights(cfg, 12)
    toks = tokens(48, cfg["vocab"], 13)
    want = Ref(cfg, w).forward(toks)
    gpu = S.gpu_model(cfg, w, "bfloat16")
    try:
        got = gpu.step([(0, toks)], list(range(48)))
        e = np.array([S.rel_err(got[i], want[i]) for i in range(48)])
        assert np.median(e) < BF16_TOL / 2 and (e < BF16_TOL).mean() > 0.95
    finally:
        gpu.close()


@pytest.mark.parametrize("layers,width,taps,loop", [
    ([S.latent(heads=1, dim=10, rot_dim=6, vdim=7, kv_rank=18, mlp=S.dense(9))], 40, 2, None),                 # sizes no vector load takes
    ([S.latent(heads=5, dim=4, rot_dim=2, vdim=3, kv_rank=17, mlp=S.moe(experts=3, top=2, ff=5, shared_ff=7))], 37, 3, (0, 1, 2)),   # odd everywhere
    ([S.latent(heads=2, dim=40, rot_dim=24, vdim=72, kv_rank=136, mlp=S.moe(experts=2, top=1, ff=4, shared_ff=4))], 72, 4, None),
    ([S.latent(heads=9, dim=16, rot_dim=16, vdim=8, kv_rank=64, mlp=S.dense(136))], 48, 2, None),             # heads beyond one group of eight
    ([S.latent(heads=17, dim=8, rot_dim=8, vdim=16, kv_rank=24)], 32, 3, (0, 1, 3)),
    ([S.latent(heads=2, dim=8, rot_dim=0, vdim=8, kv_rank=16, mlp=S.dense(8))], 32, 4, None),                  # nothing rotated
    ([S.latent(heads=2, dim=16, rot_dim=16, vdim=24, kv_rank=300, mlp=S.moe(experts=9, top=4, ff=12, shared_ff=20))], 56, 6, None),   # wide latent
])
@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_other_sizes(b200, layers, width, taps, loop, compute):
    cfg = S.config(layers, width=width, vocab=50, taps=taps, loop=loop, eps=3e-4)
    tol = F32_TOL if compute == "float32" else BF16_TOL
    w = S.random_weights(cfg, 13)
    toks = tokens(33, cfg["vocab"], 14)
    want = Ref(cfg, w).forward(toks)
    gpu = S.gpu_model(cfg, w, compute)
    try:
        got = gpu.step([(0, toks[:26])], list(range(26)))
        assert np.median([S.rel_err(got[i], want[i]) for i in range(26)]) < tol
        if compute == "float32":
            assert S.rel_err(got, want[:26]) < tol
        rest = decoded(gpu, toks[26:])
        assert np.median([S.rel_err(rest[i], want[26 + i]) for i in range(7)]) < tol
        if compute == "float32":
            assert S.rel_err(rest, want[26:]) < tol
    finally:
        gpu.close()


# ---------------------------------------------------------------------------------------------------- prompts, portions, batches
def test_prompt_against_token_by_token(b200):
    cfg = full_cfg()
    w = S.random_weights(cfg, 19)
    toks = tokens(34, cfg["vocab"], 20)
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
    # rings and cached rows of every pass have to carry over the cuts; portions below the number of taps leave older inputs in the ring
    cfg = full_cfg()
    w = S.random_weights(cfg, 21)
    toks = tokens(37, cfg["vocab"], 22)
    want = Ref(cfg, w).forward(toks)
    for compute, tol in (("float32", F32_TOL), ("bfloat16", BF16_TOL)):
        gpu = S.gpu_model(cfg, w, compute)
        try:
            got = []
            for a in range(0, len(toks), portion):
                part = toks[a:a + portion]
                got.append(gpu.step([(1, part)], list(range(len(part)))))
            assert S.rel_err(np.concatenate(got), want) < tol
        finally:
            gpu.close()


def test_portions_between_decoded_tokens(b200):
    # prompts, single tokens and short portions in turn: the decoding kernels and the prompt kernels share one ring
    cfg = full_cfg()
    w = S.random_weights(cfg, 23)
    cuts = [1, 1, 2, 1, 5, 1, 1, 1, 3, 9, 1, 2, 2, 20, 1]
    toks = tokens(sum(cuts), cfg["vocab"], 24)
    want = Ref(cfg, w).forward(toks)
    gpu = S.gpu_model(cfg, w)
    try:
        got, a = [], 0
        for n in cuts:
            got.append(gpu.step([(2, toks[a:a + n])], list(range(n))))
            a += n
        assert S.rel_err(np.concatenate(got), want) < F32_TOL
    finally:
        gpu.close()


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_unequal_batch_against_each_alone(b200, compute):
    tol = F32_TOL if compute == "float32" else BF16_TOL
    cfg = full_cfg()
    w = S.random_weights(cfg, 25)
    ref = Ref(cfg, w)
    prompts = [tokens(n, cfg["vocab"], 20 + n) for n in (1, 13, 29, 6)]
    tails = [tokens(9, cfg["vocab"], 40 + i) for i in range(4)]
    gpu = S.gpu_model(cfg, w, compute, max_batch=6)
    try:
        slots = [4, 0, 2, 5]
        got = gpu.step(list(zip(slots, prompts)), list(range(sum(len(p) for p in prompts))))
        at, states = 0, []
        for p in prompts:
            st = ref.new()
            assert S.rel_err(got[at:at + len(p)], ref.step(st, p)) < tol
            states.append(st)
            at += len(p)
        for k in range(9):                                          # the shortest request ends first, then the next one
            alive = [i for i in range(4) if k < 3 + 2 * i]
            lg = gpu.decode_batch([slots[i] for i in alive], [tails[i][k] for i in alive])
            for j, i in enumerate(alive):
                assert S.rel_err(lg[j], ref.step(states[i], [tails[i][k]])[0]) < tol, (k, i)
    finally:
        gpu.close()


def test_mixed_batch_of_prompts_and_single_tokens(b200):
    cfg = full_cfg()
    w = S.random_weights(cfg, 26)
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


@pytest.mark.parametrize("rows", [2, 3, 5, 8, 11, 16, 24, 40])
def test_decoding_many_sequences(b200, rows):
    # every row count the few-row kernels are built for, and the counts beyond them
    cfg = S.config([S.latent(mlp=S.moe()), S.latent(heads=10, mlp=S.dense())], taps=3, loop=(0, 1, 2))
    w = S.random_weights(cfg, 27)
    ref = Ref(cfg, w)
    seqs = [tokens(3 + (5 * i) % 7, cfg["vocab"], 100 + i) for i in range(rows)]
    tails = [tokens(3, cfg["vocab"], 200 + i) for i in range(rows)]
    for compute, tol in (("float32", F32_TOL), ("bfloat16", BF16_TOL)):
        gpu = S.gpu_model(cfg, w, compute, max_batch=rows, max_seq_len=32)
        try:
            gpu.step([(i, t) for i, t in enumerate(seqs)])
            got = [gpu.decode_batch(list(range(rows)), [t[k] for t in tails]) for k in range(3)]
            errs = []
            for i in range(rows):
                want = ref.forward(seqs[i] + tails[i])[len(seqs[i]):]
                errs += [S.rel_err(got[k][i], want[k]) for k in range(3)]
            assert np.median(errs) < tol / 2 and (compute == "bfloat16" or max(errs) < tol)
        finally:
            gpu.close()


def test_slots_freed_and_used_again(b200):
    cfg = full_cfg()
    w = S.random_weights(cfg, 28)
    ref = Ref(cfg, w)
    gpu = S.gpu_model(cfg, w, max_batch=3)
    try:
        assert gpu.pool_counts() == (0, 0)
        a, b, c = tokens(30, cfg["vocab"], 3), tokens(18, cfg["vocab"], 4), tokens(25, cfg["vocab"], 5)
        gpu.step([(0, a), (1, b)])
        assert gpu.pool_counts() == (2, 0)
        gpu.reset(0)
        assert gpu.pool_counts() == (1, 1) and gpu.position(0) == 0
        # slot 2 takes the block that slot 0 left (full of a's rows and inputs); slot 1 goes on undisturbed
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
def planted_key_model(rows_wide=False):
    """One latent-attention layer in which the probe token's queries point at the needle token's latent.  Fewer tokens than the width and
    one tap: a vector g with g . h = 1 for the needle's mixer input and 0 for every other token's exists, and W_dkv + (big u) g^T gives the
    needle alone the latent direction u, the mean direction of the probe's queries carried into the latent.  Its score stands out among
    hundreds of random ones in every head (the shared rotated key part is scaled down for that)."""
    extra = dict(kv_rank=160, rot_dim=32) if rows_wide else dict(kv_rank=32, rot_dim=16)
    cfg = S.config([S.latent(heads=2, dim=16, vdim=24, scale=1.0, **extra)], width=48, vocab=40, taps=1)
    w = S.random_weights(cfg, 29)
    w["l0.mix.dkv.norm"] = np.ones_like(w["l0.mix.dkv.norm"])
    w["l0.mix.g"] = 0.2 * w["l0.mix.g"]
    needle, probe = cfg["vocab"] - 2, cfg["vocab"] - 1
    W, eps = S.f64(w), cfg["norm"]["eps"]
    m = cfg["layers"][0]["mixer"]
    hin = []
    for t in range(cfg["vocab"]):
        x = O.scalar_norm(W["embed"][t], W["embed.norm"], eps)
        hin.append(O.input_convolution(O.scalar_norm(x, W["l0.norm1"], eps), W["l0.canon1"], O.Delay(1, cfg["width"])))
    hin = np.stack(hin)
    g = np.linalg.pinv(hin)[:, needle]
    assert np.abs(hin @ g - np.eye(cfg["vocab"])[needle]).max() < 1e-9
    q = (W["l0.mix.q"] @ hin[probe]).reshape(m["heads"], m["dim"] + m["rot_dim"])
    uk = W["l0.mix.uk"].reshape(m["heads"], m["dim"], m["kv_rank"])
    qa = np.stack([uk[h].T @ q[h, :m["dim"]] for h in range(m["heads"])])
    u = (qa / np.linalg.norm(qa, axis=1, keepdims=True)).sum(axis=0)
    u /= np.linalg.norm(u)
    d = np.array(w["l0.mix.dkv"], dtype=np.float64)
    d[:m["kv_rank"]] += np.outer(60.0 * u, g)
    d[m["kv_rank"]:] *= 0.2
    w["l0.mix.dkv"] = d.astype(np.float32)
    return cfg, w, needle, probe


@pytest.mark.parametrize("rows_wide", [False, True])
def test_far_key_among_hundreds(b200, rows_wide):
    # probes from position 290 on, in a prompt and decoded, meet a needle at the very start, at the borders of the kernels' key tiles and
    # in between
    cfg, w, needle, probe = planted_key_model(rows_wide)
    n, cut = 304, 297
    ref = Ref(cfg, w)
    base = tokens(n, cfg["vocab"] - 2, 30)
    base[290:] = [probe] * (n - 290)
    plain = ref.forward(base)
    for at in ((0, 31, 64) if rows_wide else (0, 1, 31, 32, 63, 64, 127, 200)):
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


def edge_cfg(taps):
    return S.config([S.latent(heads=2, mlp=S.dense(24))], width=48, vocab=64, taps=taps)


@pytest.mark.parametrize("taps", [2, 3, 4, 6])
def test_input_convolution_edges(b200, taps):
    # The oldest tap carries the largest weight: whether the input taps - 1 places back (just inside) or taps places back (just outside) is
    # meant shows at every position, in prompts, portions cut anywhere, and decoding from the first token on.
    cfg = edge_cfg(taps)
    w = S.random_weights(cfg, 31)
    for c in ("l0.canon1", "l0.canon2"):
        w[c] = np.array(w[c])
        w[c][:, 0] = 2.0
    n = 40
    toks = tokens(n, cfg["vocab"], 32)
    ref = Ref(cfg, w)
    want = ref.forward(toks)
    shifted = {k: (np.roll(v, 1, axis=1) if ".canon" in k else v) for k, v in w.items()}
    assert min(S.rel_err(a, b) for a, b in zip(Ref(cfg, shifted).forward(toks)[taps:], want[taps:])) > 50 * F32_TOL
    for compute, tol in (("float32", F32_TOL), ("bfloat16", BF16_TOL)):
        gpu = S.gpu_model(cfg, w, compute)
        try:
            assert S.rel_err(gpu.step([(0, toks)], list(range(n))), want) < tol
            for cut in range(1, 12):
                got = np.concatenate([gpu.step([(1, toks[:cut])], list(range(cut))), gpu.step([(1, toks[cut:])], list(range(n - cut)))])
                assert S.rel_err(got, want) < tol, cut
                gpu.reset(1)
            assert S.rel_err(decoded(gpu, toks, seq=2), want) < tol
        finally:
            gpu.close()


def test_first_tokens_and_long_decoding(b200):
    cfg = full_cfg()
    w = S.random_weights(cfg, 33)
    toks = tokens(140, cfg["vocab"], 34)      # decoded one by one from the very first token, over several key tiles
    want = Ref(cfg, w).forward(toks)
    gpu = S.gpu_model(cfg, w)
    try:
        got = decoded(gpu, toks)
        for p in range(len(toks)):
            assert S.rel_err(got[p], want[p]) < F32_TOL, p
    finally:
        gpu.close()


def test_rotation_at_large_positions(b200):
    # a small base makes every pair turn many times; positions beyond 1500 in a prompt and decoded
    cfg = S.config([S.latent(heads=2, dim=8, rot_dim=16, vdim=16, base=4.0)], width=32, vocab=40, taps=2)
    w = S.random_weights(cfg, 35)
    n = 1556
    toks = tokens(n, cfg["vocab"], 36)
    want = Ref(cfg, w).forward(toks)
    gpu = S.gpu_model(cfg, w, max_seq_len=n + 4)
    try:
        assert S.rel_err(gpu.step([(0, toks[:1550])], list(range(1500, 1550))), want[1500:1550]) < F32_TOL
        assert S.rel_err(decoded(gpu, toks[1550:]), want[1550:]) < F32_TOL
    finally:
        gpu.close()


def test_row_does_not_depend_on_the_batch(b200):
    cfg = full_cfg()
    w = S.random_weights(cfg, 37)
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
    w = S.random_weights(cfg, 38)
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
    w = S.random_weights(cfg, 39)
    p = tokens(12, cfg["vocab"], 40)
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
    from llama_gguf_b200 import fizesun

    cfg = full_cfg()
    w = S.random_weights(cfg, 41)
    short = dict(w)
    del short["l2.mlp.shared.sg"]
    with pytest.raises(b200.InvalidArgument):
        S.gpu_model(cfg, short)
    wrong = dict(w)
    wrong["l1.norm1"] = np.ones(cfg["width"], dtype=np.float32)      # a weight per coordinate where one number belongs
    with pytest.raises(b200.ShapeMismatch):
        S.gpu_model(cfg, wrong)
    program, layers = fizesun.parse_config(cfg, 64, 2, "float32")
    for bad in (dict(program, in_conv=65), dict(program, streams=2), dict(program, parallel_ff=1), dict(program, loop_stop=0)):
        with pytest.raises(b200.InvalidArgument):
            b200.LayerProgramInference(bad, layers, {})
    bad = copy.deepcopy(layers)
    bad[0]["moe"]["limit"] = 0.0
    with pytest.raises(b200.InvalidArgument):
        b200.LayerProgramInference(program, bad, {})


# ---------------------------------------------------------------------------------------------------- kernels against their plain forms
@pytest.mark.parametrize("sizes", [(3, 16, 32), (1, 16, 48), (5, 32, 96), (3, 8, 40), (7, 64, 192), (2, 64, 256)])
def test_tile_attention_against_warp_attention(b200, monkeypatch, sizes):
    # bf16 prompts of 16 rows and more take the tensor-pipe tile kernel when the cached row is a multiple of 16 wide (fourth case: it is not,
    # both runs take the warp kernel; last two: the wide instantiation); B200_LP_ATTN_TILE=0 keeps the warp kernel
    heads, rot_dim, kv_rank = sizes
    cfg = S.config([S.latent(heads=heads, dim=16, rot_dim=rot_dim, vdim=24, kv_rank=kv_rank)], width=64, vocab=64, taps=2)
    w = S.random_weights(cfg, 42)
    a, b = tokens(190, cfg["vocab"], 43), tokens(70, cfg["vocab"], 44)
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
    # (the tile kernel rounds queries and rows to bf16: a row whose weight hangs on one or two keys differs most)
    d = np.array([S.rel_err(x, y) for x, y in zip(out["1"], out["0"])])
    assert S.rel_err(out["1"], want[37:]) < BF16_TOL
    assert np.median(d) < 1e-2 and d.max() < BF16_TOL / 2


def test_tensor_core_gemm_path(b200, monkeypatch):
    # bf16 steps of 17 rows and more multiply on the tensor cores, the per-head products and the experts' grouped products included
    cfg = full_cfg()
    w = S.random_weights(cfg, 45)
    toks = tokens(200, cfg["vocab"], 46)
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
    e = np.array([S.rel_err(out["1"][i], want[i]) for i in range(len(toks))])
    assert np.median(e) < BF16_TOL / 2


@pytest.mark.parametrize("env", [{}, {"B200_LP_FUSE": "0"}, {"B200_LP_LAT_SPLIT": "0"}, {"B200_LP_CONV_FUSE_ROWS": "0"}, {"B200_LP_CONV_FUSE_ROWS": "8"},
                                 {"B200_LP_GRAPH": "0"}, {"B200_LP_FUSE": "0", "B200_LP_GRAPH": "0"}])
def test_decode_kernels_against_the_unfused_forms(b200, monkeypatch, env):
    cfg = full_cfg()
    w = S.random_weights(cfg, 47)
    ref = Ref(cfg, w)
    prompts = [tokens(n, cfg["vocab"], 60 + n) for n in (3, 19, 1)]
    tails = [tokens(12, cfg["vocab"], 70 + i) for i in range(3)]
    states = [ref.new() for _ in prompts]
    for st, pr in zip(states, prompts):
        ref.step(st, pr)
    want = [[ref.step(states[i], [tails[i][k]])[0] for i in range(3)] for k in range(12)]
    for k, v in env.items():
        monkeypatch.setenv(k, v)
    gpu = S.gpu_model(cfg, w, "float32")
    try:
        gpu.step([(i, pr) for i, pr in enumerate(prompts)])
        for k in range(12):
            lg = gpu.decode_batch([0, 1, 2], [tails[i][k] for i in range(3)])
            for i in range(3):
                assert S.rel_err(lg[i], want[k][i]) < F32_TOL, (k, i)
    finally:
        gpu.close()


@pytest.mark.parametrize("rows", [3, 7, 9, 16])
def test_small_batches_on_the_tensor_pipe(b200, monkeypatch, rows):
    # bf16 steps of 3 to 16 rows: products with K a multiple of 32 run on mma.sync (here every one; output counts that no tile of 16 divides
    # included), and rows that choose more experts than there are take every expert once; B200_LP_GEMV_MMA=0 keeps the CUDA-core kernels
    cfg = S.config([S.latent(heads=3, dim=16, rot_dim=8, vdim=32, mlp=S.moe(experts=4, top=2, ff=32, shared_ff=64)), S.latent(heads=2, vdim=16, mlp=S.dense(96))],
                   width=96, vocab=101, taps=3, loop=(0, 1, 2))
    w = S.random_weights(cfg, 48)
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


def test_trace_runner_on_a_model_folder(b200, tmp_path):
    # config.json + model.safetensors (bf16) on disk -> registry -> bin/trace_run: two requests start together with unequal prompts, are
    # decoded together, the shorter one ends first; logits of the wanted rows come back in files
    import json
    import os
    import subprocess
    import sys

    from llama_gguf_b200.safetensors_io import bf16_bits, write_safetensors

    cfg = full_cfg()
    w = S.random_weights(cfg, 51)
    d = tmp_path / "model"
    d.mkdir()
    (d / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(d / "model.safetensors"), {n: bf16_bits(a).reshape(a.shape) for n, a in w.items()})
    a, b = tokens(19, cfg["vocab"], 52), tokens(7, cfg["vocab"], 53)
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
