"""A plain float64 restatement of the Gefovik design, one function per mechanism, one token at a time.  It shares nothing with the
library: the tests compare the library's logits and residual streams with what these functions give.

Notation.  h: a sublayer's input vector (the residual stream itself); W[name]: a tensor of the model, linear maps stored [out, in] and
applied as W @ h; p: the token's position in its sequence, counted from 0."""
import math

import numpy as np


def layer_norm(x, w, eps):
    """Mean off, over the root of the mean squared deviation, times a weight per coordinate; no bias."""
    d = x - x.mean()
    return d / math.sqrt((d * d).mean() + eps) * w


def unit_rms(x, eps):
    """x over its root mean square."""
    return x / math.sqrt((x * x).mean() + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def temperature(p, coef, every):
    """What a query at position p is multiplied by: one more `coef` for every e-fold of finished spans of `every` positions."""
    return 1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0)


def cap(s, limit):
    return limit * np.tanh(s / limit)


class Rows:
    """What one layer keeps of the earlier tokens: one array per name, a row per position."""

    def __init__(self, names):
        self.n = 0
        self.data = dict.fromkeys(names)

    def append(self, **rows):
        for name, x in rows.items():
            old = self.data[name]
            if old is None or self.n == len(old):
                new = np.zeros((max(16, 2 * self.n),) + np.shape(x))
                if self.n:
                    new[:self.n] = old[:self.n]
                self.data[name] = old = new
            old[self.n] = x
        self.n += 1

    def upto(self, name):
        return self.data[name][:self.n]


def attention(h, p, W, pre, mx, eps, rows):
    """One token.  A key is the projected key over its root mean square, its value the projected key as it is."""
    H, G, dim = mx["heads"], mx["kv_heads"], mx["dim"]
    q = (W[pre + "q"] @ h).reshape(H, dim)
    k = (W[pre + "k"] @ h).reshape(G, dim)
    rows.append(k=np.array([unit_rms(x, eps) for x in k]), v=k)
    assert rows.n == p + 1
    t = temperature(p, mx["q_temp"]["coef"], mx["q_temp"]["every"])
    out = np.zeros((H, dim))
    for n in range(H):
        g = n // (H // G)
        s = cap(rows.upto("k")[:, g] @ (unit_rms(q[n], eps) * t) * mx["scale"], mx["softcap"])
        a = np.exp(s - s.max())
        out[n] = (a / a.sum()) @ rows.upto("v")[:, g]
    return W[pre + "o"] @ out.reshape(-1)


def latent_attention(h, p, W, pre, mx, eps, rows):
    """One token.  Keys and values are read out of the latent position by position and head by head (no absorbed products)."""
    H, dim, vd = mx["heads"], mx["dim"], mx["vdim"]
    q = (W[pre + "q"] @ h).reshape(H, dim)
    c = unit_rms(W[pre + "dkv"] @ h, eps) * W[pre + "dkv.norm"]
    rows.append(k=(W[pre + "uk"] @ c).reshape(H, dim), v=(W[pre + "uv"] @ c).reshape(H, vd))
    assert rows.n == p + 1
    gate = sigmoid(W[pre + "g"] @ h)
    out = np.zeros((H, vd))
    for n in range(H):
        s = rows.upto("k")[:, n] @ q[n] * mx["scale"]
        sink = float(W[pre + "sink"][n])
        top = max(s.max(), sink)
        a = np.exp(s - top)
        out[n] = gate[n] * ((a / (a.sum() + math.exp(sink - top))) @ rows.upto("v")[:, n])
    return W[pre + "o"] @ out.reshape(-1)


def relu_unit(h, W, pre):
    return W[pre + "down"] @ (np.maximum(W[pre + "gate"] @ h, 0.0) * (W[pre + "up"] @ h))


def silu_unit(h, W, pre):
    z = W[pre + "gate"] @ h
    return W[pre + "down"] @ (z * sigmoid(z) * (W[pre + "up"] @ h))


def routing(h, W, pre):
    """-> (softmax over all outputs of the router, the same plus the correction)"""
    z = W[pre + "router"] @ h
    s = np.exp(z - z.max())
    s /= s.sum()
    return s, s + W[pre + "correction"]


def expert_mixture(h, W, pre, mlp):
    """The corrected scores decide who is chosen, the scores alone with what weight; the outputs behind the experts' stand for the input
    itself."""
    r = mlp["router"]
    s, choice = routing(h, W, pre)
    out = np.zeros_like(h)
    for e in sorted(range(len(s)), key=lambda e: (-choice[e], e))[:r["top"]]:
        out = out + s[e] * (silu_unit(h, W, pre + "e%d." % e) if e < r["experts"] else h)
    return out


def sublayer_step(x, y, w, eps):
    """The stream after a sublayer gave y."""
    return x + layer_norm(y, w, eps)


class Sequence:
    """One sequence fed token by token."""

    def __init__(self, cfg, W):
        self.cfg, self.W, self.p = cfg, W, 0
        self.margin = math.inf          # the closest call of any choice so far
        self.rows = [Rows(("k", "v")) for _ in cfg["layers"]]

    def token(self, tok):
        """-> (logits [vocab], the residual stream after every layer [layers, width])"""
        cfg, W, eps = self.cfg, self.W, self.cfg["norm"]["eps"]
        x = W["embed"][tok] * cfg["embedding"]["scale"]
        taps = []
        for i, L in enumerate(cfg["layers"]):
            pre = "l%d." % i
            mix = attention if L["type"] == "attention" else latent_attention
            x = sublayer_step(x, mix(x, self.p, W, pre + "mix.", L["mixer"], eps, self.rows[i]), W[pre + "norm1"], eps)
            mlp = L.get("mlp")
            if mlp is not None and mlp["kind"] == "moe":
                c = np.append(np.sort(routing(x, W, pre + "mlp.")[1])[::-1], -math.inf)
                self.margin = min(self.margin, c[mlp["router"]["top"] - 1] - c[mlp["router"]["top"]])
            if mlp is not None:
                ff = relu_unit(x, W, pre + "mlp.") if mlp["kind"] == "dense" else expert_mixture(x, W, pre + "mlp.", mlp)
                x = sublayer_step(x, ff, W[pre + "norm2"], eps)
            taps.append(x)
        self.p += 1
        return W["embed"] @ layer_norm(x, W["final.norm"], eps), np.array(taps)


def run(cfg, W, tokens):
    """-> logits [n, vocab], taps [layers, n, width]"""
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
