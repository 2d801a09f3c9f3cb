"""Plain numpy statement of the layered designs, one function per mechanism, token by token and in float64.

Slow on purpose and independent of the product: nothing here imports tl_b200.  A model is (cfg, weights) with cfg the dict of
config.json and weights a dict name -> array.  Every mixer carries its history in a dict `st` it owns, so a sequence can be
fed in any portions: forward(model, tokens, state) returns the logits of the new tokens.
"""
import numpy as np


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_zero_centred(x, w, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return unit_rms(x, eps) * (1.0 + w)


def poly_norm(z, coef, eps):
    """sum over the powers 1..3 of coef * (z^n over its own root mean square), plus a constant."""
    a, b, c, e = coef
    return a * unit_rms(z, eps) + b * unit_rms(z * z, eps) + c * unit_rms(z ** 3, eps) + e


def rotate_half(x, pos, base, dims):
    """x [heads, dim]; dimension i turns with i + dims/2 by pos * base^(-2i/dims), the dimensions past dims stay."""
    half = dims // 2
    ang = pos * np.power(float(base), -2.0 * np.arange(half) / dims)
    c, s = np.cos(ang), np.sin(ang)
    u, v = x[:, :half], x[:, half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[:, dims:]], axis=1)


def attention_token(q, ks, vs, scale, r1, r2, sink, window):
    """One query against its history.  q [H, d]; ks [T, G, d], vs [T, G, dv] with the query's own token last."""
    T, G = ks.shape[0], ks.shape[1]
    H = q.shape[0]
    first = max(0, T - window)
    out = np.zeros((H, vs.shape[2]))
    for h in range(H):
        g = h // (H // G)
        dist = (T - 1) - np.arange(first, T)
        s = ks[first:, g] @ q[h] * scale - r1[h] * np.log(1.0 + r2[h] * dist)
        m = max(np.max(s), sink[h])
        e = np.exp(s - m)
        out[h] = e @ vs[first:, g] / (np.sum(e) + np.exp(sink[h] - m))
    return out


def retention_token(S, q, k, v, decay):
    """S [H, d, dv] -> new S and o [H, dv]."""
    S = decay[:, None, None] * S + k[:, :, None] * v[:, None, :]
    return S, np.einsum("hdv,hd->hv", S, q)


def general_delta_token(S, r, k, v, w, a):
    """One step of the generalised delta rule per head; S [H, d, d] is indexed [key channel, value channel]."""
    u = k / np.sqrt(np.sum(k * k, axis=-1, keepdims=True) + 1e-6)
    seen = np.einsum("hd,hdv->hv", u, S)
    S = w[:, :, None] * S - (a * u)[:, :, None] * seen[:, None, :] + k[:, :, None] * v[:, None, :]
    return S, np.einsum("hdv,hd->hv", S, r)


def delta_decay(h, w1, w2, w0):
    return np.exp(-np.exp(-0.5) * sigmoid(w2 @ np.tanh(w1 @ h) + w0))


class Plain:
    def __init__(self, cfg, weights):
        self.cfg = cfg
        self.w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
        self.eps = cfg["norm"]["eps"]

    def new_state(self):
        return {"pos": 0, "layers": [dict() for _ in self.cfg["layers"]]}

    def mixer(self, i, h, pos, st):
        lay = self.cfg["layers"][i]
        m, t = lay["mixer"], lay["type"]
        W = lambda n: self.w["l%d.mix.%s" % (i, n)]
        H, d = m["heads"], m["dim"]
        if t == "attention":
            G, dv = m["kv_heads"], m["vdim"]
            q = (W("q") @ h + W("q.b")).reshape(H, d)
            st.setdefault("k", []).append((W("k") @ h + W("k.b")).reshape(G, d))
            st.setdefault("v", []).append((W("v") @ h + W("v.b")).reshape(G, dv))
            o = attention_token(q, np.stack(st["k"]), np.stack(st["v"]), m["scale"], W("r1"), W("r2"), W("sink"), m["mask"]["size"])
            return W("o") @ o.reshape(-1)
        if t == "retention":
            dv, rot = m["vdim"], m["rot"]
            q = rotate_half((W("q") @ h).reshape(H, d), pos, rot["base"], rot["dims"])
            k = rotate_half((W("k") @ h).reshape(H, d), pos, rot["base"], rot["dims"]) * d ** -0.5
            v = (W("v") @ h).reshape(H, dv)
            S = st.get("S", np.zeros((H, d, dv)))
            st["S"], o = retention_token(S, q, k, v, np.asarray(m["decay"], dtype=np.float64))
            return W("o") @ (unit_rms(o, self.eps).reshape(-1) * silu(W("g") @ h))
        if t == "general_delta":
            r, k, v = ((W(n) @ h).reshape(H, d) for n in "rkv")
            w = delta_decay(h, W("w1"), W("w2"), W("w0")).reshape(H, d)
            a = sigmoid(W("a") @ h + W("a.b")).reshape(H, d)
            S = st.get("S", np.zeros((H, d, d)))
            st["S"], o = general_delta_token(S, r, k, v, w, a)
            return W("o") @ (unit_rms(o, self.eps).reshape(-1) * W("norm") * sigmoid(W("g") @ h))
        raise ValueError(t)

    def token(self, tok, state, layers_out=None):
        x = self.w["embed"][tok]
        for i, lay in enumerate(self.cfg["layers"]):
            p = "l%d." % i
            x = x + self.w[p + "ls1"] * self.mixer(i, norm_zero_centred(x, self.w[p + "norm1"], self.eps), state["pos"], state["layers"][i])
            if lay.get("mlp") is not None:
                z = self.w[p + "mlp.up"] @ norm_zero_centred(x, self.w[p + "norm2"], self.eps)
                x = x + self.w[p + "ls2"] * (self.w[p + "mlp.down"] @ poly_norm(z, self.w[p + "mlp.act"], self.eps))
            if layers_out is not None:
                layers_out[i].append(x)
        state["pos"] += 1
        return self.w["head"] @ norm_zero_centred(x, self.w["final.norm"], self.eps)

    def forward(self, tokens, state, layers_out=None):
        return np.stack([self.token(int(t), state, layers_out) for t in tokens])
