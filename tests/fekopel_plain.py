"""The Fekopel design in plain numpy float64: one function per mechanism, whole sequences at once, no cache and no state.
It is the oracle of the Fekopel tests and shares no code with the product.

Notation: T tokens, width W; a mixer has H heads over G key heads of size D with values of size Dv.  Matrices are stored
[out, in]; `h @ M.T` applies M to every row of h."""
import math

import numpy as np


# ------------------------------------------------------------------------------------------------ small pieces
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def gelu_erf(z):
    """z times the standard normal distribution function at z."""
    return 0.5 * z * (1.0 + np.vectorize(math.erf, otypes=[np.float64])(z / math.sqrt(2.0)))


def layer_norm(x, w, b, eps):
    mean = x.mean(axis=-1, keepdims=True)
    var = ((x - mean) ** 2).mean(axis=-1, keepdims=True)
    return (x - mean) / np.sqrt(var + eps) * w + b


def rms_unit(x, eps):
    """x over the root of (its mean square + eps), along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def softmax(z):
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


# ------------------------------------------------------------------------------------------------ attention
def visible(T, window, keep=0):
    """[T, T] bool: query i sees j <= i among the last `window` positions (0: all of them) or the first `keep` ones."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    v = j <= i
    if window:
        v &= (i - j < window) | (j < keep)
    return v


def rotate_halves(x, positions, rot):
    """x [T, heads, D]: coordinate i < dims / 2 is paired with i + dims / 2; the pair turns by position * base^(-2 i / dims)."""
    if not rot or not rot.get("dims"):
        return x
    d = rot["dims"]
    f = rot["base"] ** (-2.0 * np.arange(d // 2) / d)
    ang = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    a, b = x[..., :d // 2], x[..., d // 2:d]
    return np.concatenate([a * c - b * s, b * c + a * s, x[..., d:]], axis=-1)


def sink_softmax(s, sink=None):
    """soft-max along the last axis; with a sink one more exp(sink) in the denominator that no value goes with."""
    m = s.max(axis=-1, keepdims=True)
    if sink is not None:
        m = np.maximum(m, sink)
    e = np.exp(s - m)
    total = e.sum(axis=-1, keepdims=True)
    return e / (total if sink is None else total + np.exp(sink - m))


def attention_core(q, k, v, scale, vis, softcap=0.0, sink=None):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] (normed and rotated already) -> [T, H, Dv]; sink: a score per head or None."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if softcap:
            s = softcap * np.tanh(s / softcap)
        s = np.where(vis, s, -np.inf)
        out[:, h] = sink_softmax(s, None if sink is None else sink[h]) @ v[:, g]
    return out


def project_heads(h, W, p, m):
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    return (h @ W[p + "q"].T).reshape(T, H, D), (h @ W[p + "k"].T).reshape(T, G, D), (h @ W[p + "v"].T).reshape(T, G, Dv)


def attention_sink(h, W, p, m, eps):
    """No positions; unit q and k; a sliding window; a sink of score 0."""
    T = h.shape[0]
    q, k, v = project_heads(h, W, p, m)
    o = attention_core(rms_unit(q, eps), rms_unit(k, eps), v, m["scale"], visible(T, (m.get("mask") or {}).get("size", 0)), sink=np.zeros(m["heads"]))
    return o.reshape(T, -1) @ W[p + "o"].T


def attention_gated(h, W, p, m, eps):
    """Weighted norms of q and k per head, rotary halves, soft-capped scores, a window that keeps the first positions, a sigmoid
    gate per element."""
    T = h.shape[0]
    q, k, v = project_heads(h, W, p, m)
    pos, mask = np.arange(T), m.get("mask") or {}
    q = rotate_halves(rms_unit(q, eps) * W[p + "q.norm"], pos, m.get("rot"))
    k = rotate_halves(rms_unit(k, eps) * W[p + "k.norm"], pos, m.get("rot"))
    o = attention_core(q, k, v, m["scale"], visible(T, mask.get("size", 0), mask.get("keep_first", 0)), softcap=m.get("softcap", 0.0))
    return (o.reshape(T, -1) * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def expert(h, up, down):
    return gelu_erf(h @ up.T) @ down.T


def route(h, router, top, groups=1, keep=1, scale=1.0):
    """-> (chosen experts [T, top], weights [T, top]): soft-max over all experts; the `keep` groups of neighbours that hold the
    largest scores stay; the weights are the chosen scores over their sum, times scale."""
    s = softmax(h @ router.T)
    T, E = s.shape
    best = s.reshape(T, groups, E // groups).max(axis=-1)
    stay = np.argsort(-best, axis=-1, kind="stable")[:, :keep]
    masked = np.full_like(s, -np.inf).reshape(T, groups, E // groups)
    for t in range(T):
        masked[t, stay[t]] = s[t].reshape(groups, -1)[stay[t]]
    order = np.argsort(-masked.reshape(T, E), axis=-1, kind="stable")[:, :top]
    w = np.take_along_axis(s, order, axis=-1)
    return order, w / (w.sum(axis=-1, keepdims=True) + 1e-20) * scale


def route_margin(h, router, top, groups=1, keep=1):
    """How far in logits the choice of every token is from another one: the last group that stays to the first that goes, the last
    expert chosen to the first that is not."""
    z = h @ router.T
    T, E = z.shape
    best = z.reshape(T, groups, E // groups).max(axis=-1)
    order = np.argsort(-best, axis=-1, kind="stable")
    gap = np.full(T, np.inf)
    cand = z.reshape(T, groups, E // groups).copy()
    if keep < groups:
        rows = np.arange(T)
        gap = best[rows, order[:, keep - 1]] - best[rows, order[:, keep]]
        for t in range(T):
            cand[t, order[t, keep:]] = -np.inf
    ranked = -np.sort(-cand.reshape(T, E), axis=-1)
    if top < E:
        gap = np.minimum(gap, ranked[:, top - 1] - ranked[:, top])
    return gap


def moe_ff(h, W, p, f, margins=None):
    r = f["router"]
    g = r.get("groups") or {}
    count = g.get("count", 1)
    idx, wt = route(h, W[p + "router"], r["top"], count, g.get("keep", count), r.get("scale", 1.0))
    if margins is not None:
        margins.append(route_margin(h, W[p + "router"], r["top"], count, g.get("keep", count)))
    out = np.zeros_like(h)
    for e in np.unique(idx):
        t, slot = np.nonzero(idx == e)
        out[t] += wt[t, slot][:, None] * expert(h[t], W[p + "e%d.up" % e], W[p + "e%d.down" % e])
    if f.get("shared"):
        out += sigmoid(h @ W[p + "shared.sg"].T) * expert(h, W[p + "shared.up"], W[p + "shared.down"])
    return out


# ------------------------------------------------------------------------------------------------ the model
def layer_runs(cfg):
    """(layer, number of the pass that begins with this run or None) in order."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp or lp["stop"] <= lp["start"]:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(lp["start"])]
    for t in range(lp["times"]):
        runs += [(i, t if i == lp["start"] else None) for i in range(lp["start"], lp["stop"])]
    return runs + [(i, None) for i in range(lp["stop"], n)]


MIXERS = {"attention": attention_sink, "attention_2": attention_gated}


def forward(tokens, W, cfg, layers_out=None, margins=None):
    """Logits [T, vocab] of a whole sequence; layers_out collects the residual after every layer run, margins every router's."""
    eps = cfg["norm"]["eps"]
    x0 = W["embed"][np.asarray(tokens)].astype(np.float64)
    x = x0.copy()

    def norm(x, name):
        return layer_norm(x, W[name], W[name + ".b"], eps)

    for li, step in layer_runs(cfg):
        L, p = cfg["layers"][li], "l%d." % li
        if step is not None:
            x = x + (x0 if step > 0 else 0.0) + W["loop.step"][step]
        x = x + MIXERS[L["type"]](norm(x, p + "norm1"), W, p + "mix.", L["mixer"], eps)
        if L.get("mlp"):
            x = x + moe_ff(norm(x, p + "norm2"), W, p + "mlp.", L["mlp"], margins)
        if layers_out is not None:
            layers_out.append(x)
    return norm(x, "final.norm") @ W["head"].T


# ------------------------------------------------------------------------------------------------ random weights
def random_weights(cfg, seed=0):
    """name -> float64 array, sized so that activations stay of order one through the layers."""
    r = np.random.default_rng(seed)
    Wd, V = cfg["width"], cfg["vocab"]
    W = {"embed": r.standard_normal((V, Wd)), "head": r.standard_normal((V, Wd)) / np.sqrt(Wd)}

    def mat(n_out, n_in, gain=1.0):
        return gain * r.standard_normal((n_out, n_in)) / np.sqrt(n_in)

    def norm(name, n=Wd):
        W[name], W[name + ".b"] = 1.0 + 0.1 * r.standard_normal(n), 0.2 * r.standard_normal(n)

    norm("final.norm")
    if cfg.get("loop"):
        W["loop.step"] = 0.5 * r.standard_normal((cfg["loop"]["times"], Wd))
    for li, L in enumerate(cfg["layers"]):
        p, m = "l%d." % li, L["mixer"]
        H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        norm(p + "norm1")
        W[p + "mix.q"], W[p + "mix.k"], W[p + "mix.v"], W[p + "mix.o"] = mat(H * D, Wd), mat(G * D, Wd), mat(G * Dv, Wd), mat(Wd, H * Dv)
        if L["type"] == "attention_2":
            W[p + "mix.q.norm"], W[p + "mix.k.norm"] = 1.0 + 0.3 * r.standard_normal(D), 1.0 + 0.3 * r.standard_normal(D)
            W[p + "mix.g"] = mat(H * Dv, Wd, 1.5)
        f = L.get("mlp")
        if f:
            norm(p + "norm2")
            E, ff = f["router"]["experts"], f["expert"]["ff"]
            W[p + "mlp.router"] = mat(E, Wd, 2.0)
            for e in range(E):
                W[p + "mlp.e%d.up" % e], W[p + "mlp.e%d.down" % e] = mat(ff, Wd, 1.5), mat(Wd, ff)
            if f.get("shared"):
                fs = f["shared"]["ff"]
                W[p + "mlp.shared.up"], W[p + "mlp.shared.down"], W[p + "mlp.shared.sg"] = mat(fs, Wd, 1.5), mat(Wd, fs), mat(1, Wd, 1.5)
    return W
