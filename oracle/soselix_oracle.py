"""A slow float64 restatement of the Soselix design, one token at a time, one function per mechanism.

It shares nothing with the CUDA path: plain numpy on the tensors of a checkpoint, every sequence advanced token by
token through explicit per-layer state objects (lists of past latents, carried convolution inputs, recurrent matrices).

Notation.  x is the residual of one token, m the residual multiplier, N_g(x) = g x / sqrt(mean(x^2) + eps) with ONE
number g.  A layer does

    x <- x + m mixer(N_g1(x)),    x <- x + m ff(N_g2(x))        (the second line only where the layer has a feed-forward)

Mixers: latent attention (queries through a normed latent, keys and values rebuilt from one cached latent per token, a
sink in the denominator, one output gate per head; a layer may read the cached latents of an earlier layer), the HGRN2
recurrence (the forget gate also decides what is written), and Mamba-2 (a scalar decay per head and token, keys and
queries shared by the heads of a group).  Feed-forward: one biased hidden layer under xIELU.
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


def rotate_half(v, p, rot):
    """Rotate the first rot['dims'] entries of every row of v [rows, n] by position p; entry i pairs with i + dims/2."""
    n = (rot or {}).get("dims", 0)
    if not n:
        return v
    half = n // 2
    ang = p * float(rot["base"]) ** (-2.0 * np.arange(half) / n)
    c, s = np.cos(ang), np.sin(ang)
    out = np.array(v, dtype=np.float64, copy=True)
    a, b = v[..., :half], v[..., half:n]
    out[..., :half] = a * c - b * s
    out[..., half:n] = b * c + a * s
    return out


def sink_softmax(scores, sink):
    """Weights of the given scores when the denominator also holds exp(sink)."""
    m = max(np.max(scores), sink)
    e = np.exp(scores - m)
    return e / (e.sum() + np.exp(sink - m))


class CarriedConv:
    """Causal convolution over time per channel: y_t = b + sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""

    def __init__(self, w, b):
        self.w, self.b = w, b
        self.past = [np.zeros(w.shape[0]) for _ in range(w.shape[1] - 1)]

    def step(self, u):
        seq = self.past + [u]
        y = self.b + sum(self.w[:, j] * seq[j] for j in range(self.w.shape[1]))
        self.past = seq[1:]
        return y


class LatentCache:
    """What a layer keeps per token: the normed latent and the rotated key part that all heads share."""

    def __init__(self):
        self.c, self.kr = [], []

    def write(self, P, mx, h, eps):
        C = mx["kv_rank"]
        d = P["dkv"] @ h
        self.c.append(unit_rms(d[:C], eps) * P["dkv.norm"])
        self.kr.append(rotate_half(d[C:][None], len(self.kr), mx.get("rot"))[0])


class LatentAttention:
    """Per head: score_j = (q . W_uk c_j + rot(q') . k'_j) * scale, softmax with a sink, W_uv on the sum, gate, W_o."""

    def __init__(self, P, mx, eps, shared=None):
        self.P, self.mx, self.eps = P, mx, eps
        self.cache = LatentCache() if shared is None else shared
        self.own = shared is None
        self.p = 0

    def queries(self, h):
        """(unrotated [heads, dim], rotated [heads, rot_dim]) of the token at position self.p."""
        P, mx = self.P, self.mx
        cq = unit_rms(P["dq"] @ h, self.eps) * P["dq.norm"]
        q = (P["uq"] @ cq).reshape(mx["heads"], mx["dim"] + mx["rot_dim"])
        return q[:, :mx["dim"]], rotate_half(q[:, mx["dim"]:], self.p, mx.get("rot"))

    def step(self, h):
        P, mx = self.P, self.mx
        H, D, Dv = mx["heads"], mx["dim"], mx["vdim"]
        if self.own:
            self.cache.write(P, mx, h, self.eps)
        qn, qr = self.queries(h)
        self.p += 1
        c, kr = np.stack(self.cache.c[:self.p]), np.stack(self.cache.kr[:self.p])       # keys 0 .. own position
        uk, uv = P["uk"].reshape(H, D, -1), P["uv"].reshape(H, Dv, -1)
        gate = sigmoid(P["g"] @ h)
        out = np.zeros((H, Dv))
        for hd in range(H):
            s = ((c @ uk[hd].T) @ qn[hd] + kr @ qr[hd]) * mx["scale"]
            out[hd] = gate[hd] * (sink_softmax(s, P["sink"][hd]) @ (c @ uv[hd].T))
        return P["o"] @ out.reshape(-1)


def forget_gate(z, lower):
    """(f, 1 - f) with f = lower + (1 - lower) sigmoid(z); the second is formed without a subtraction from 1."""
    return lower + (1.0 - lower) * sigmoid(z), (1.0 - lower) * sigmoid(-z)


class Hgrn2:
    """S <- diag(f) S + (1 - f) v^T, o = S^T q per head; every head's o RMS-normed with one shared weight."""

    def __init__(self, P, mx, eps):
        self.P, self.mx, self.eps = P, mx, eps
        self.S = np.zeros((mx["heads"], mx["dim"], mx["vdim"]))

    def step(self, h):
        P, mx = self.P, self.mx
        H, D, Dv = mx["heads"], mx["dim"], mx["vdim"]
        q = silu(P["q"] @ h).reshape(H, D)
        v = (P["v"] @ h).reshape(H, Dv)
        f, w = forget_gate(P["f"] @ h + P["f.b"], P["lower"])
        f, w = f.reshape(H, D), w.reshape(H, D)
        self.S = f[:, :, None] * self.S + w[:, :, None] * v[:, None, :]
        o = np.einsum("hdv,hd->hv", self.S, q)
        return P["o"] @ (unit_rms(o, self.eps) * P["norm"]).reshape(-1)


def grouped_gated_norm(y, z, groups, w, eps):
    """silu gate first, then every one of `groups` equal parts divided by its own root mean square, then the weight."""
    u = (y * silu(z)).reshape(groups, -1)
    return unit_rms(u, eps).reshape(-1) * w


class Mamba2:
    """S <- exp(-exp(A_log) d) S + d B x^T, y = S^T C + D x per head, B and C shared by the heads of a group."""

    def __init__(self, P, mx, eps):
        self.P, self.mx, self.eps = P, mx, eps
        self.conv = CarriedConv(P["conv"], P["conv.b"])
        self.S = np.zeros((mx["heads"], mx["state"], mx["vdim"]))

    def step(self, h):
        P, mx = self.P, self.mx
        H, Dv, N, G = mx["heads"], mx["vdim"], mx["state"], mx["groups"]
        I = H * Dv
        u = P["in"] @ h
        z, xbc, dt = u[:I], silu(self.conv.step(u[I:2 * I + 2 * G * N])), u[2 * I + 2 * G * N:]
        x, B, C = xbc[:I].reshape(H, Dv), xbc[I:I + G * N].reshape(G, N), xbc[I + G * N:].reshape(G, N)
        d = softplus(dt + P["dt_bias"])
        y = np.zeros((H, Dv))
        for hd in range(H):
            g = hd // (H // G)
            self.S[hd] = np.exp(-np.exp(P["A_log"][hd]) * d[hd]) * self.S[hd] + d[hd] * np.outer(B[g], x[hd])
            y[hd] = self.S[hd].T @ C[g] + P["D"][hd] * x[hd]
        return P["o"] @ grouped_gated_norm(y.reshape(-1), z, mx["norm_groups"], P["norm"], self.eps)


def xielu(z, p, q):
    """z > 0: softplus(p) z^2 + z / 2;   z <= 0: (1/2 + softplus(q)) (exp(z) - 1 - z) + z / 2."""
    neg = np.minimum(z, 0.0)
    return np.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (np.expm1(neg) - neg)) + 0.5 * z


def dense_ff(P, h):
    return P["down"] @ xielu(P["up"] @ h + P["up.b"], P["act"][0], P["act"][1]) + P["down.b"]


def sub(P, prefix):
    return {k[len(prefix):]: v for k, v in P.items() if k.startswith(prefix)}


class SoselixOracle:
    def __init__(self, cfg, W):
        self.cfg = cfg
        self.W = {k: np.asarray(v, dtype=np.float64) for k, v in W.items()}
        self.eps = cfg["norm"]["eps"]
        self.mlp = [sub(self.W, "l%d.mlp." % i) if L.get("mlp") else None for i, L in enumerate(cfg["layers"])]

    def new_state(self):
        out = []
        for i, L in enumerate(self.cfg["layers"]):
            P, mx = sub(self.W, "l%d.mix." % i), L["mixer"]
            if L["type"] == "latent_attention":
                j = mx.get("kv_from")
                out.append(LatentAttention(P, mx, self.eps, None if j is None else out[j].cache))
            else:
                out.append({"hgrn2": Hgrn2, "mamba2": Mamba2}[L["type"]](P, mx, self.eps))
        return out

    def norm(self, name, x):
        return unit_rms(x, self.eps) * float(self.W[name])

    def step(self, state, token, layers_out=None):
        """Advance one sequence by one token; returns its logits."""
        m = self.cfg["residual_mult"]
        x = self.W["embed"][token] * self.cfg["embedding"]["scale"]
        for i, mixer in enumerate(state):
            x = x + m * mixer.step(self.norm("l%d.norm1" % i, x))
            if self.mlp[i] is not None:
                x = x + m * dense_ff(self.mlp[i], self.norm("l%d.norm2" % i, x))
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
