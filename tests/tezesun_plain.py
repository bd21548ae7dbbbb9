"""The Tezesun design in plain numpy float64: one function per mechanism, whole sequences at once, no cache and no state.
It is the oracle of the Tezesun tests and shares no code with the product.

Notation: T tokens, width W; an attention has H query heads over G key / value heads, keys of size D, values of size Dv.
Matrices are stored [out, in]; `h @ M.T` applies M to every row of h."""
import numpy as np


# ------------------------------------------------------------------------------------------------ small pieces
def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def rms_unit(x, eps):
    """x over the root of (its mean square + eps), along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return rms_unit(x, eps) * w


def softmax(z):
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


# ------------------------------------------------------------------------------------------------ the layer's frame
def token_shift(h, mu):
    """Per channel a blend between the token's own row and the one before it (zeros before the first)."""
    before = np.concatenate([np.zeros((1, h.shape[1])), h[:-1]], axis=0)
    return h + (before - h) * mu


def xielu(z, p, q):
    """Positive side quadratic, negative side exponential, both plus z / 2; p and q pass a softplus."""
    neg = np.minimum(z, 0.0)
    return np.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (np.expm1(neg) - neg)) + 0.5 * z


def dense_ff(h, up, down, act):
    return xielu(h @ up.T, act[0], act[1]) @ down.T


# ------------------------------------------------------------------------------------------------ rotary positions
def rot_frequencies(rot):
    """(frequencies [dims / 2], magnitude): plain, or blended between plain and divided ones over a ramp of turns."""
    d, base = rot["dims"], rot["base"]
    i = np.arange(d // 2)
    f = base ** (-2.0 * i / d)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def dim_of(turns):
        return d * np.log(sc["original"] / (2.0 * np.pi * turns)) / (2.0 * np.log(base))
    lo, hi = max(np.floor(dim_of(sc["fast"])), 0.0), min(np.ceil(dim_of(sc["slow"])), d - 1.0)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * np.log(sc["factor"]) + 1.0


def rotate(x, positions, rot, halves):
    """x [T, heads, D]: the first `dims` coordinates turn in pairs (2i, 2i + 1), or with `halves` (i, i + dims / 2)."""
    if not rot or not rot.get("dims"):
        return x
    d = rot["dims"]
    f, mag = rot_frequencies(rot)
    ang = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = mag * np.cos(ang)[:, None, :], mag * np.sin(ang)[:, None, :]
    y = x.copy()
    a, b = (slice(0, d // 2), slice(d // 2, d)) if halves else (slice(0, d, 2), slice(1, d, 2))
    y[..., a] = x[..., a] * c - x[..., b] * s
    y[..., b] = x[..., b] * c + x[..., a] * s
    return y


# ------------------------------------------------------------------------------------------------ differential attention
def visible(T, size, keep_first=0, pos0=0):
    """[T, T] bool: query i sees key j <= i among the last `size` positions (0: all) or among the first keep_first."""
    i = np.arange(pos0, pos0 + T)[:, None]
    j = np.arange(pos0, pos0 + T)[None, :]
    v = j <= i
    if size:
        v &= (i - j < size) | (j < keep_first)
    return v


def attention_map(q, k, v, scale, softcap, vis):
    """one soft-max attention: q [T, D], k [T, D], v [T, Dv] -> [T, Dv]"""
    s = (q @ k.T) * scale
    if softcap:
        s = softcap * np.tanh(s / softcap)
    return softmax(np.where(vis, s, -np.inf)) @ v


def diff_lambda(lq1, lk1, lq2, lk2, diff):
    return np.exp(np.sum(lq1 * lk1)) - np.exp(np.sum(lq2 * lk2)) + diff


def diff_core(q, k, v, scale, softcap, vis, lam, diff, eps):
    """q [T, H, 2, D], k [T, G, 2, D] (already rotated), v [T, G, Dv] -> [T, H, Dv]: the second map's output, times lam,
    taken from the first one's; divided by its root mean square; times 1 - diff."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        a = [attention_map(q[:, h, m], k[:, g, m], v[:, g], scale, softcap, vis) for m in (0, 1)]
        out[:, h] = rms_unit(a[0] - lam * a[1], eps) * (1.0 - diff)
    return out


def diff_attention(h, W, p, m, eps):
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"]
    pos = np.arange(T)
    q = rotate((h @ W[p + "q"].T).reshape(T, 2 * H, D), pos, m.get("rot"), False).reshape(T, H, 2, D)
    k = rotate((h @ W[p + "k"].T).reshape(T, 2 * G, D), pos, m.get("rot"), False).reshape(T, G, 2, D)
    v = (h @ W[p + "v"].T).reshape(T, G, Dv)
    mask = m.get("mask") or {}
    lam = diff_lambda(W[p + "lq1"], W[p + "lk1"], W[p + "lq2"], W[p + "lk2"], m["diff"])
    o = diff_core(q, k, v, m["scale"], m.get("softcap", 0.0), visible(T, mask.get("size", 0), mask.get("keep_first", 0)), lam, m["diff"], eps)
    return (o.reshape(T, H * Dv) * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------------ latent attention
def latent_attention(h, W, p, m, eps):
    T = h.shape[0]
    H, D, Dr, Dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    q = (rms_norm(h @ W[p + "dq"].T, W[p + "dq.norm"], eps) @ W[p + "uq"].T).reshape(T, H, D + Dr)
    qr = rotate(q[..., D:], pos, m.get("rot"), True)
    d = h @ W[p + "dkv"].T
    c = rms_norm(d[:, :R], W[p + "dkv.norm"], eps)
    kr = rotate(d[:, None, R:], pos, m.get("rot"), True)[:, 0]
    ku, v = (c @ W[p + "uk"].T).reshape(T, H, D), (c @ W[p + "uv"].T).reshape(T, H, Dv)
    vis = visible(T, 0)
    o = np.zeros((T, H, Dv))
    for i in range(H):
        s = (q[:, i, :D] @ ku[:, i].T + qr[:, i] @ kr.T) * m["scale"]
        o[:, i] = softmax(np.where(vis, s, -np.inf)) @ v[:, i]
    return o.reshape(T, H * Dv) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------------ gated linear recurrence
def causal_conv(x, w, b):
    """x [T, C], w [C, taps]: y[t] = b + sum_j w[:, j] x[t - (taps - 1) + j], zeros before the start."""
    T, C = x.shape
    taps = w.shape[1]
    xx = np.concatenate([np.zeros((taps - 1, C)), x], axis=0)
    return sum(xx[j:j + T] * w[:, j][None, :] for j in range(taps)) + b


def block_product(u, w, b):
    """u [T, C] cut into blocks of d; w [blocks, d, d] as [out, in] per block, b [blocks, d] -> [T, C]"""
    nb, d = b.shape
    return np.stack([u[:, i * d:(i + 1) * d] @ w[i].T + b[i] for i in range(nb)], axis=1).reshape(u.shape)


def rglru_core(u, r, i, lam, S0=None):
    """u, r, i [T, C] (the two gates after their sigmoid) -> (S [T, C], last S): S <- a S + sqrt(1 - a^2) i u with
    a = exp(-8 r softplus(lam))."""
    S = np.zeros(u.shape[1]) if S0 is None else S0.copy()
    out = np.zeros(u.shape)
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * softplus(lam)
        S = np.exp(log_a) * S + np.sqrt(-np.expm1(2.0 * log_a)) * i[t] * u[t]
        out[t] = S
    return out, S


def rglru(h, W, p, m):
    y = gelu_tanh(h @ W[p + "y"].T + W[p + "y.b"])
    u = causal_conv(h @ W[p + "x"].T + W[p + "x.b"], W[p + "conv"], W[p + "conv.b"])
    r, i = sigmoid(block_product(u, W[p + "ra"], W[p + "ra.b"])), sigmoid(block_product(u, W[p + "ri"], W[p + "ri.b"]))
    return (rglru_core(u, r, i, W[p + "lam"])[0] * y) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------------ the model
def forward(tokens, W, cfg, layers_out=None):
    """Logits [T, vocab] of a whole sequence; layers_out collects the residual after every layer."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens, dtype=np.int64)].astype(np.float64)
    for li, L in enumerate(cfg["layers"]):
        p, m = "l%d." % li, L["mixer"]
        h = rms_norm(x, W[p + "norm1"], eps)
        hs = token_shift(h, W[p + "shift"])
        if L["type"] == "attention":
            y = diff_attention(hs, W, p + "mix.", m, eps)
        elif L["type"] == "latent_attention":
            y = latent_attention(hs, W, p + "mix.", m, eps)
        else:
            y = rglru(hs, W, p + "mix.", m)
        y = y * W[p + "ls1"]
        if L.get("mlp"):
            y = y + dense_ff(h, W[p + "mlp.up"], W[p + "mlp.down"], W[p + "mlp.act"]) * W[p + "ls2"]
        x = x + y
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, W["final.norm"], eps) @ W["head"].T * cfg["logit_scale"]


# ------------------------------------------------------------------------------------------------ random weights
def random_weights(cfg, seed=0):
    """name -> float64 array, sized so that activations stay of order one through the layers."""
    r = np.random.default_rng(seed)
    Wd, V = cfg["width"], cfg["vocab"]

    def mat(n_out, n_in, gain=1.0):
        return gain * r.standard_normal((n_out, n_in)) / np.sqrt(n_in)

    W = {"embed": r.standard_normal((V, Wd)), "head": 2.0 * mat(V, Wd), "final.norm": 1.0 + 0.1 * r.standard_normal(Wd)}
    for li, L in enumerate(cfg["layers"]):
        p, m = "l%d." % li, L["mixer"]
        W[p + "norm1"] = 1.0 + 0.1 * r.standard_normal(Wd)
        W[p + "ls1"] = 0.8 + 0.2 * r.standard_normal(Wd)
        W[p + "shift"] = r.uniform(0.0, 1.0, Wd)
        q = p + "mix."
        if L["type"] == "attention":
            H, G, D, Dv = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"]
            W[q + "q"], W[q + "k"], W[q + "v"] = mat(2 * H * D, Wd, 2.0), mat(2 * G * D, Wd, 2.0), mat(G * Dv, Wd)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                W[q + n] = 0.4 * r.standard_normal(D) / D ** 0.25
            W[q + "g"], W[q + "o"] = mat(H * Dv, Wd), mat(Wd, H * Dv)
        elif L["type"] == "latent_attention":
            H, D, Dr, Dv, R, Rq = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            W[q + "dq"], W[q + "dq.norm"], W[q + "uq"] = mat(Rq, Wd), 1.0 + 0.1 * r.standard_normal(Rq), mat(H * (D + Dr), Rq, 2.0)
            W[q + "dkv"], W[q + "dkv.norm"] = mat(R + Dr, Wd, 1.5), 1.0 + 0.1 * r.standard_normal(R)
            W[q + "uk"], W[q + "uv"], W[q + "o"] = mat(H * D, R, 1.5), mat(H * Dv, R), mat(Wd, H * Dv)
        else:
            C, nb, taps = m["width"], m["blocks"], m["conv"]
            d = C // nb
            W[q + "y"], W[q + "x"] = mat(C, Wd), mat(C, Wd)
            for n in ("y.b", "x.b", "conv.b", "lam"):
                W[q + n] = 0.5 * r.standard_normal(C)
            W[q + "conv"] = 0.6 * r.standard_normal((C, taps))
            for n in ("ra", "ri"):
                W[q + n] = r.standard_normal((nb, d, d)) / np.sqrt(d)
                W[q + n + ".b"] = r.standard_normal((nb, d)) - (1.5 if n == "ra" else 0.0)
            W[q + "lam"] -= 2.5
            W[q + "o"] = mat(Wd, C)
        if L.get("mlp"):
            W[p + "ls2"] = 0.8 + 0.2 * r.standard_normal(Wd)
            W[p + "mlp.up"], W[p + "mlp.down"] = mat(L["mlp"]["ff"], Wd), mat(Wd, L["mlp"]["ff"])
            W[p + "mlp.act"] = r.standard_normal(2)
    return W
