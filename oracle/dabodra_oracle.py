"""A slow float64 restatement of the Dabodra design, one token at a time, one function per mechanism.

It shares nothing with the CUDA path: plain numpy on the tensors of a checkpoint, every sequence advanced token by
token through explicit per-layer state objects (lists of past keys and values, carried convolution inputs, matrices).

Notation.  x is the residual of one token, N_w(u) = u / sqrt(mean(u^2) + eps) * (1 + w).  The residual starts at
N(embed[token]) and a sublayer reads it as it is, only its output is normed:

    x <- x + N_1(mixer(x)),    x <- x + N_2(ff(x))        (the second only where the layer has a feed-forward)

Mixers: sliding-window softmax attention whose values are the projected keys and whose denominator has a sink, and the
gated delta rule (a decayed matrix memory that writes only the difference to what it already holds under the key).
Feed-forward: sigmoid-scored experts, eligible by groups, beside a shared expert.
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return np.exp(-np.logaddexp(0.0, -np.asarray(z, dtype=np.float64)))      # no overflow, small values keep their digits


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def unit_rms(v, eps):
    """v / sqrt(mean(v^2) + eps) over the last axis."""
    v = np.asarray(v, dtype=np.float64)
    return v / np.sqrt((v * v).mean(axis=-1, keepdims=True) + eps)


def unit_length(v):
    """v / sqrt(sum(v^2) + 1e-6) over the last axis."""
    return v / np.sqrt((v * v).sum(axis=-1, keepdims=True) + 1e-6)


def rotate_pairs(v, p, rot):
    """Rotate the first rot['dims'] entries of every row of v [rows, n] by position p; entry 2i pairs with 2i + 1."""
    n = (rot or {}).get("dims", 0)
    if not n:
        return v
    ang = p * float(rot["base"]) ** (-2.0 * np.arange(n // 2) / n)
    c, s = np.cos(ang), np.sin(ang)
    out = np.array(v, dtype=np.float64, copy=True)
    a, b = v[..., 0:n:2], v[..., 1:n:2]
    out[..., 0:n:2] = a * c - b * s
    out[..., 1:n:2] = b * c + a * s
    return out


def sink_softmax(scores, sink):
    """Weights of the given scores when the denominator also holds exp(sink)."""
    m = max(np.max(scores), sink)
    e = np.exp(scores - m)
    return e / (e.sum() + np.exp(sink - m))


def window_start(p, size):
    """First position the token at position p sees."""
    return max(0, p - size + 1)


class WindowAttention:
    """score_j = (rot(norm(q)) . rot(norm(k_j))) * scale over the window, softmax with a sink, values = unnormed k_j."""

    def __init__(self, P, mx, eps):
        self.P, self.mx, self.eps = P, mx, eps
        self.k, self.v = [], []

    def project(self, h, p):
        """(queries [heads, dim], keys [kv_heads, dim], values [kv_heads, dim]) of a token; q and k normed as whole rows."""
        P, mx = self.P, self.mx
        q, k = P["q"] @ h, P["k"] @ h
        qn = (unit_rms(q, self.eps) * P["q.norm"]).reshape(mx["heads"], mx["dim"])
        kn = (unit_rms(k, self.eps) * P["k.norm"]).reshape(mx["kv_heads"], mx["dim"])
        return rotate_pairs(qn, p, mx["rot"]), rotate_pairs(kn, p, mx["rot"]), k.reshape(mx["kv_heads"], mx["vdim"])

    def step(self, h):
        P, mx = self.P, self.mx
        p = len(self.k)
        q, k, v = self.project(h, p)
        self.k.append(k)
        self.v.append(v)
        lo = window_start(p, mx["mask"]["size"])
        keys, vals = np.stack(self.k[lo:]), np.stack(self.v[lo:])
        per = mx["heads"] // mx["kv_heads"]
        out = np.zeros((mx["heads"], mx["vdim"]))
        for hd in range(mx["heads"]):
            out[hd] = sink_softmax(keys[:, hd // per] @ q[hd] * mx["scale"], P["sink"][hd]) @ vals[:, hd // per]
        return P["o"] @ out.reshape(-1)


class CarriedConv:
    """Causal convolution over time per channel: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""

    def __init__(self, w):
        self.w = w
        self.past = [np.zeros(w.shape[0]) for _ in range(w.shape[1] - 1)]

    def step(self, u):
        seq = self.past + [u]
        y = sum(self.w[:, j] * seq[j] for j in range(self.w.shape[1]))
        self.past = seq[1:]
        return y


def delta_gates(P, h):
    """(beta, g) per head: the step size and the decay of this token."""
    return sigmoid(P["b"] @ h), np.exp(-np.exp(P["A_log"]) * softplus(P["a"] @ h + P["dt_bias"]))


def delta_update(S, g, beta, q, k, v):
    """One head: decay, write beta times what v differs from the memory's answer to k, read with q.  Returns (S, o)."""
    S = g * S
    S = S + np.outer(k, beta * (v - S.T @ k))
    return S, S.T @ q


class GatedDelta:
    def __init__(self, P, mx, eps):
        self.P, self.mx, self.eps = P, mx, eps
        self.conv = {n: CarriedConv(P[n + ".conv"]) for n in "qkv"}
        self.S = np.zeros((mx["heads"], mx["dim"], mx["vdim"]))

    def step(self, h):
        P, mx = self.P, self.mx
        H, G, D, Dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
        q, k, v = (silu(self.conv[n].step(P[n] @ h)) for n in "qkv")
        q, k = unit_length(q.reshape(G, D)) * D ** -0.5, unit_length(k.reshape(G, D))
        v = v.reshape(H, Dv)
        beta, g = delta_gates(P, h)
        o = np.zeros((H, Dv))
        for hd in range(H):
            kv = hd // (H // G)
            self.S[hd], o[hd] = delta_update(self.S[hd], g[hd], beta[hd], q[kv], k[kv], v[hd])
        return P["o"] @ (unit_rms(o, self.eps) * P["norm"] * silu(P["g"] @ h).reshape(H, Dv)).reshape(-1)


def route(s, correction, router):
    """(chosen experts, weights) from the scores s = sigmoid(z): ranked by s + correction inside the best groups only."""
    c = s + correction
    gr = router.get("groups") or dict(count=1, keep=1)
    parts = c.reshape(gr["count"], -1)
    rank = np.sort(parts, axis=1)[:, -2:].sum(axis=1)
    open_ = np.zeros(len(s), dtype=bool)
    for g in np.argsort(-rank, kind="stable")[:gr["keep"]]:
        open_[g * parts.shape[1]:(g + 1) * parts.shape[1]] = True
    pick = np.argsort(-np.where(open_, c, -np.inf), kind="stable")[:router["top"]]
    return pick, s[pick] / (s[pick].sum() + 1e-20) * router["scale"]


def gated_ff(P, h):
    return P["down"] @ (silu(P["gate"] @ h) * (P["up"] @ h))


def experts_ff(P, mlp, h):
    pick, w = route(sigmoid(P["router"] @ h), P["correction"], mlp["router"])
    y = sum(wi * gated_ff(sub(P, "e%d." % e), h) for e, wi in zip(pick, w))
    return y + gated_ff(sub(P, "shared."), h) if mlp.get("shared") else y


def sub(P, prefix):
    return {k[len(prefix):]: v for k, v in P.items() if k.startswith(prefix)}


class DabodraOracle:
    def __init__(self, cfg, W):
        self.cfg = cfg
        self.W = {k: np.asarray(v, dtype=np.float64) for k, v in W.items()}
        self.eps = cfg["norm"]["eps"]
        self.mlp = [sub(self.W, "l%d.mlp." % i) if L.get("mlp") else None for i, L in enumerate(cfg["layers"])]

    def new_state(self):
        return [{"attention": WindowAttention, "delta": GatedDelta}[L["type"]](sub(self.W, "l%d.mix." % i), L["mixer"], self.eps)
                for i, L in enumerate(self.cfg["layers"])]

    def norm(self, name, x):
        return unit_rms(x, self.eps) * (1.0 + self.W[name])

    def step(self, state, token, layers_out=None):
        """Advance one sequence by one token; returns its logits."""
        x = self.norm("embed.norm", self.W["embed"][token])
        for i, mixer in enumerate(state):
            x = x + self.norm("l%d.norm1" % i, mixer.step(x))
            if self.mlp[i] is not None:
                x = x + self.norm("l%d.norm2" % i, experts_ff(self.mlp[i], self.cfg["layers"][i]["mlp"], x))
            if layers_out is not None:
                layers_out.append(x)
        return self.W["head"] @ self.norm("final.norm", x)

    def forward(self, tokens, return_layers=False):
        """Logits of every position [T, vocab]; with return_layers also the residual after every layer."""
        state = self.new_state()
        logits, per_tok = [], []
        for t in tokens:
            lo = []
            logits.append(self.step(state, int(t), lo))
            per_tok.append(lo)
        if return_layers:
            return np.stack(logits), np.stack(per_tok, axis=1)
        return np.stack(logits)

    def generate(self, prompt, n):
        """Greedy continuation: (tokens, smallest top-1 / top-2 margin met on the way)."""
        state = self.new_state()
        lg = None
        for t in prompt:
            lg = self.step(state, int(t))
        out, margin = [], float("inf")
        for _ in range(n):
            top = np.sort(lg)[-2:]
            margin = min(margin, top[1] - top[0])
            out.append(int(np.argmax(lg)))
            lg = self.step(state, out[-1])
        return out, margin
