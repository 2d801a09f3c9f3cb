"""Plain numpy statement of the Rukedra design, one function per mechanism, token by token and in float64.

Slow on purpose and independent of the product: nothing here imports tl_b200.  A model is (cfg, weights) as in plain_layers.py, and
a sequence can be fed in any portions: forward(tokens, state) returns the logits of the new tokens.
"""
import math

import numpy as np

from plain_layers import sigmoid, silu, unit_rms


def grouped_rms(x, w, groups, eps):
    """Consecutive parts of x, each over its own root mean square; then the weight of every element."""
    return unit_rms(x.reshape(groups, -1), eps).reshape(-1) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotation_speeds(dims, base, scaling=None):
    """(radians per position of every pair, factor on cosine and sine).  With scaling, pairs that turn fewer than `slow` times in
    `original` positions are slowed down by `factor`, those that turn more than `fast` times keep their speed, a ramp between."""
    i = np.arange(dims // 2)
    f = np.power(float(base), -2.0 * i / dims)
    if scaling is None:
        return f, 1.0
    where = lambda turns: dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(where(scaling["fast"])), 0), min(math.ceil(where(scaling["slow"])), dims - 1)
    slow = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return slow * f / scaling["factor"] + (1.0 - slow) * f, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_pairs(x, pos, speeds, gain):
    """x [..., 2 n]: every pair of neighbours as a complex number, turned by its angle and stretched."""
    z = (x[..., 0::2] + 1j * x[..., 1::2]) * gain * np.exp(1j * pos * speeds)
    out = np.empty_like(x)
    out[..., 0::2], out[..., 1::2] = z.real, z.imag
    return out


def softmax(s):
    e = np.exp(s - np.max(s))
    return e / np.sum(e)


def attend(q, keys, values, scale, window=None):
    """One query per head against its history.  q [H, d]; keys [T, H, d] and values [T, H, dv] with the query's own token last."""
    first = 0 if window is None else max(0, len(keys) - window)
    return np.stack([softmax(keys[first:, h] @ q[h] * scale) @ values[first:, h] for h in range(len(q))])


def min_gru_token(S, z, u, zb, xb):
    """z, u: the projections without their biases."""
    g, v = sigmoid(z + zb), u + xb
    return (1.0 - g) * S + g * np.where(v >= 0, v + 0.5, sigmoid(v))


def choose_experts(logits, top, groups, keep, scale):
    """(experts, weights) of one token."""
    s = sigmoid(logits)
    parts = np.sort(s.reshape(groups, -1), axis=1)
    best = np.argsort(-parts[:, -2:].sum(axis=1), kind="stable")[:keep]
    masked = np.where(np.isin(np.arange(len(s)) // (len(s) // groups), best), s, -np.inf)
    pick = np.argsort(-masked, kind="stable")[:top]
    return pick, s[pick] / (np.sum(s[pick]) + 1e-20) * scale


def choice_margin(logits, top, groups, keep):
    """How far a token is from another choice: the gap behind the last group kept and the last expert chosen."""
    s = sigmoid(logits)
    parts = np.sort(s.reshape(groups, -1), axis=1)
    g = np.sort(parts[:, -2:].sum(axis=1))[::-1]
    kept = np.argsort(-parts[:, -2:].sum(axis=1), kind="stable")[:keep]
    e = np.sort(s.reshape(groups, -1)[kept].reshape(-1))[::-1]
    return min(g[keep - 1] - g[keep] if keep < groups else 1.0, e[top - 1] - e[top] if top < len(e) else 1.0)


def gated(W, p, h, act):
    return W[p + "down"] @ (act(W[p + "gate"] @ h) * (W[p + "up"] @ h))


class PlainRukedra:
    def __init__(self, cfg, weights):
        self.cfg = cfg
        self.w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
        self.eps, self.groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
        self.margins = []                   # of every choice of experts made so far

    def new_state(self):
        return {"pos": 0, "layers": [dict() for _ in self.cfg["layers"]]}

    def norm(self, x, name):
        return grouped_rms(x, self.w[name], self.groups, self.eps)

    def latent_attention(self, p, m, h, pos, st, queries_through_latent):
        W = lambda n: self.w[p + n]
        H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        if queries_through_latent:
            q = W("uq") @ (unit_rms(W("dq") @ h, self.eps) * W("dq.norm"))
        else:
            q = W("q") @ h
        q = q.reshape(H, d + r)
        speeds, gain = rotation_speeds(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
        kv = W("dkv") @ h
        c = unit_rms(kv[:R], self.eps) * W("dkv.norm")
        kr = rotate_pairs(kv[R:], pos, speeds, gain)
        st.setdefault("k", []).append(np.concatenate([(W("uk") @ c).reshape(H, d), np.tile(kr, (H, 1))], axis=1))
        st.setdefault("v", []).append((W("uv") @ c).reshape(H, dv))
        q = np.concatenate([q[:, :d], rotate_pairs(q[:, d:], pos, speeds, gain)], axis=1)
        window = m["mask"]["size"] if queries_through_latent else None
        lo = 0 if window is None else max(0, len(st["k"]) - window)
        o = attend(q, np.stack(st["k"][lo:]), np.stack(st["v"][lo:]), m["scale"], window).reshape(-1)
        if queries_through_latent:
            o = o * sigmoid(W("g") @ h)
        return W("o") @ o

    def min_gru(self, p, m, h, st):
        W = lambda n: self.w[p + n]
        S = min_gru_token(st.get("S", np.zeros(m["width"])), W("z") @ h, W("x") @ h, W("z.b"), W("x.b"))
        st["S"] = S
        return W("o") @ (S * silu(W("g") @ h))

    def feed_forward(self, p, m, h):
        if m["kind"] == "dense":
            return gated(self.w, p, h, gelu_tanh)
        r = m["router"]
        groups = r.get("groups") or {"count": 1, "keep": 1}
        z = self.w[p + "router"] @ h
        self.margins.append(choice_margin(z, r["top"], groups["count"], groups["keep"]))
        pick, weight = choose_experts(z, r["top"], groups["count"], groups["keep"], r["scale"])
        y = sum(w * gated(self.w, "%se%d." % (p, e), h, silu) for e, w in zip(pick, weight))
        if m.get("shared"):
            y = y + sigmoid(self.w[p + "shared.sg"] @ h) * gated(self.w, p + "shared.", h, silu)
        return y

    def token(self, tok, state, layers_out=None):
        x = self.w["embed"][tok]
        for i, lay in enumerate(self.cfg["layers"]):
            j = i
            while self.cfg["layers"][j].get("weights_of") is not None:
                j = self.cfg["layers"][j]["weights_of"]
            p, m, st = "l%d." % j, lay["mixer"], state["layers"][i]
            h = self.norm(x, p + "norm1")
            if lay["type"] == "mingru":
                y = self.min_gru(p + "mix.", m, h, st)
            else:
                y = self.latent_attention(p + "mix.", m, h, state["pos"], st, lay["type"] == "latent_attention")
            x = x + self.norm(y * sigmoid(self.w[p + "rg1"] @ h + self.w[p + "rg1.b"]), p + "norm1b")
            if lay.get("mlp") is not None:
                h = self.norm(x, p + "norm2")
                y = self.feed_forward(p + "mlp.", lay["mlp"], h)
                x = x + self.norm(y * sigmoid(self.w[p + "rg2"] @ h + self.w[p + "rg2.b"]), p + "norm2b")
            if layers_out is not None:
                layers_out[i].append(x)
        state["pos"] += 1
        logits = self.w["head"] @ self.norm(x, "final.norm")
        cap = self.cfg.get("logit_softcap")
        return cap * np.tanh(logits / cap) if cap else logits

    def forward(self, tokens, state, layers_out=None):
        return np.stack([self.token(int(t), state, layers_out) for t in tokens])
