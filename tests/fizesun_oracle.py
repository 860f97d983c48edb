"""A plain float64 restatement of the Fizesun design, one function per mechanism, one token at a time.  It shares nothing with the
library: the tests compare the library's logits and residual streams with what these functions give.

Notation.  h: a sublayer's input vector; W[name]: a tensor of the model, linear maps stored [out, in] and applied as W @ h;
p: the token's position in its sequence, counted from 0."""
import math

import numpy as np


def scalar_norm(x, gain, eps):
    """x over its root mean square, times ONE number for all coordinates."""
    return x / math.sqrt((x * x).mean() + eps) * float(gain)


def weighted_norm(x, w, eps):
    """x over its root mean square, times a weight per coordinate."""
    return x / math.sqrt((x * x).mean() + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0.0, z)


class Delay:
    """The last taps - 1 inputs of an input convolution, oldest first, zeros before the sequence's start."""

    def __init__(self, taps, width):
        self.past = np.zeros((taps - 1, width))


def input_convolution(h, w, delay):
    """h + sum_j w[:, j] * (h of taps - 1 - j tokens ago); w [width, taps], its last column meets the newest input."""
    window = np.vstack([delay.past, h[None, :]])
    delay.past = window[1:]
    return h + (window * w.T).sum(axis=0)


def rotate_pairs(v, p, dims, base):
    """Neighbours (2i, 2i + 1) of the first `dims` entries turn by the angle p * base^(-2i / dims)."""
    out = np.array(v, dtype=np.float64)
    for i in range(dims // 2):
        a = p * base ** (-2.0 * i / dims)
        c, s = math.cos(a), math.sin(a)
        u, t = v[2 * i], v[2 * i + 1]
        out[2 * i] = u * c - t * s
        out[2 * i + 1] = t * c + u * s
    return out


class KeyStore:
    """What one layer run keeps of the earlier tokens: per position every head's plain key and value and the shared rotated key part."""

    def __init__(self):
        self.n = 0
        self.k = self.v = self.r = None

    def append(self, k, v, r):
        if self.k is None or self.n == len(self.k):
            size = max(16, 2 * self.n)
            for name, x in (("k", k), ("v", v), ("r", r)):
                new = np.zeros((size,) + x.shape)
                if self.n:
                    new[:self.n] = getattr(self, name)[:self.n]
                setattr(self, name, new)
        self.k[self.n], self.v[self.n], self.r[self.n] = k, v, r
        self.n += 1


def latent_attention(h, p, W, pre, mx, eps, store):
    """One token.  Keys and values are read out of the latent position by position and head by head (no absorbed products)."""
    H, dim, rd, vd, rank = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    dims, base = mx["rot"]["dims"], float(mx["rot"]["base"])
    q = (W[pre + "q"] @ h).reshape(H, dim + rd)
    d = W[pre + "dkv"] @ h
    c = weighted_norm(d[:rank], W[pre + "dkv.norm"], eps)
    store.append((W[pre + "uk"] @ c).reshape(H, dim), (W[pre + "uv"] @ c).reshape(H, vd), rotate_pairs(d[rank:], p, dims, base))
    assert store.n == p + 1
    gate = sigmoid(W[pre + "g"] @ h)
    out = np.zeros((H, vd))
    for n in range(H):
        s = (store.k[:p + 1, n] @ q[n, :dim] + store.r[:p + 1] @ rotate_pairs(q[n, dim:], p, dims, base)) * mx["scale"]
        a = np.exp(s - s.max())
        out[n] = gate[n] * (a @ store.v[:p + 1, n]) / a.sum()
    return W[pre + "o"] @ out.reshape(-1)


def xielu(z, act):
    """z > 0: softplus(p) z^2 + z / 2; z <= 0: (1/2 + softplus(q)) (exp(z) - 1 - z) + z / 2, act = (p, q)."""
    a, b = softplus(float(act[0])), 0.5 + softplus(float(act[1]))
    zn = np.minimum(z, 0.0)
    return np.where(z > 0, a * z * z, b * (np.expm1(zn) - zn)) + 0.5 * z


def dense(h, W, pre):
    return W[pre + "down"] @ xielu(W[pre + "up"] @ h, W[pre + "act"])


def clamped_expert(h, gate, up, down, limit):
    g = np.minimum(gate @ h, limit)
    u = np.clip(up @ h, -limit, limit)
    return down @ (g * sigmoid(1.702 * g) * (u + 1.0))


def expert_mixture(h, W, pre, mlp):
    """The `top` largest biased logits, softmax over those alone; the shared expert with one gate per token on top."""
    r = mlp["router"]
    z = W[pre + "router"] @ h + W[pre + "router.b"]
    order = sorted(range(r["experts"]), key=lambda e: (-z[e], e))[:r["top"]]
    a = np.exp(z[order] - z[order].max())
    a /= a.sum()
    out = 0.0
    for share, e in zip(a, order):
        x = pre + "e%d." % e
        out = out + share * clamped_expert(h, W[x + "gate"], W[x + "up"], W[x + "down"], mlp["expert"]["limit"])
    if mlp.get("shared"):
        x = pre + "shared."
        out = out + sigmoid(W[x + "sg"] @ h)[0] * clamped_expert(h, W[x + "gate"], W[x + "up"], W[x + "down"], mlp["shared"]["limit"])
    return out


def enter_pass(x, x0, t, W):
    """What happens ahead of pass t of the repeated layers: a linear map of [x; x0], x0 the embedding output, plus the pass's vector."""
    return W["loop.in"] @ np.concatenate([x, x0]) + W["loop.step"][t]


def layer_runs(cfg):
    """[(layer, pass number if the run opens a pass else None)]"""
    lp = cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
    n, a, b = len(cfg["layers"]), lp["start"], lp["stop"]
    if b <= a:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(a)]
    for t in range(lp["times"]):
        out += [(i, t if i == a else None) for i in range(a, b)]
    return out + [(i, None) for i in range(b, n)]


class Sequence:
    """One sequence fed token by token."""

    def __init__(self, cfg, W):
        self.cfg, self.W, self.p = cfg, W, 0
        self.runs = layer_runs(cfg)
        taps = cfg["canon"]["taps"]
        self.keys = [KeyStore() for _ in self.runs]
        self.delay = [(Delay(taps, cfg["width"]), Delay(taps, cfg["width"])) for _ in self.runs]

    def token(self, tok):
        """-> (logits [vocab], the residual stream after every layer run [runs, width])"""
        cfg, W, eps = self.cfg, self.W, self.cfg["norm"]["eps"]
        x = x0 = scalar_norm(W["embed"][tok], W["embed.norm"], eps)
        taps = []
        for r, (i, t) in enumerate(self.runs):
            L, pre = cfg["layers"][i], "l%d." % i
            if t is not None:
                x = enter_pass(x, x0, t, W)
            h = input_convolution(scalar_norm(x, W[pre + "norm1"], eps), W[pre + "canon1"], self.delay[r][0])
            x = x + latent_attention(h, self.p, W, pre + "mix.", L["mixer"], eps, self.keys[r])
            mlp = L.get("mlp")
            if mlp is not None:
                h = input_convolution(scalar_norm(x, W[pre + "norm2"], eps), W[pre + "canon2"], self.delay[r][1])
                x = x + (dense(h, W, pre + "mlp.") if mlp["kind"] == "dense" else expert_mixture(h, W, pre + "mlp.", mlp))
            taps.append(x)
        self.p += 1
        return W["head"] @ scalar_norm(x, W["final.norm"], eps), np.array(taps)


def run(cfg, W, tokens):
    """-> logits [n, vocab], taps [layer runs, n, width]"""
    s = Sequence(cfg, W)
    out = [s.token(t) for t in tokens]
    return np.array([o[0] for o in out]), np.stack([o[1] for o in out], axis=1)


def greedy(cfg, W, prompt, n):
    """The prompt, then n tokens each the last largest logit (the library's tie rule)."""
    s = Sequence(cfg, W)
    for t in prompt:
        logits, _ = s.token(t)
    out = []
    for _ in range(n):
        t = int(np.nonzero(logits == logits.max())[0][-1])
        out.append(t)
        logits, _ = s.token(t)
    return out
