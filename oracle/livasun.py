"""Plain, slow float64 statement of the Livasun design, one function per mechanism (numpy only; test infrastructure,
never imported by the product).  It works on a whole sequence at once and keeps no cache: whatever schedule the product
runs (portions, single tokens, rings, recurrent state handed from step to step), its logits must equal these.

The stream starts as ``embed[token] * s_e``.  A layer is two pre-norm sublayers (the second is absent when the layer has no
feed-forward):

    x <- x + mixer(ln1(x));     x <- x + ff(ln2(x));        ln(x) = (x - mean) / sqrt(var + eps) * w + b

Mixers: ``mamba2`` (selective state space with one decay per head and token), ``lightning`` (linear attention with a
constant decay per head) and ``attention`` (softmax attention over a sliding window, a norm per head on queries and keys, a
query temperature that grows with the position, a bias linear in the distance, values mixed with those of the first such
layer).  Feed-forwards: dense (silu-gated) or a mixture of squared-relu experts behind a sigmoid router with a correction
and group-limited choice, plus an always-on expert.  Logits: head . ln_f(x).

Checkpoint names: ``embed``, ``head``, ``final.norm[.b]``; per layer i ``l<i>.norm1[.b]``, ``l<i>.norm2[.b]``,
``l<i>.mix.*``, ``l<i>.mlp.*``; Linear weights are [out, in].
"""
import numpy as np


def sigmoid(z):
    z = np.asarray(z, dtype=np.float64)
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * w + b


def causal_filter(u, w, b):
    """u [T, C], w [C, taps], b [C]: y_t = b + sum_j w[:, j] u_(t - taps + 1 + j), nothing before the first token."""
    taps = w.shape[1]
    past = np.concatenate([np.zeros((taps - 1, u.shape[1])), u])
    return b + sum(past[j:j + len(u)] * w[:, j] for j in range(taps))


def state_space(x, B, C, dt, a_log, D):
    """x [T, H, P], B and C [T, G, N], dt [T, H] (positive): S_t = exp(-exp(a_log) dt_t) S_(t-1) + dt_t B_t x_t^T,
    y_t = S_t^T C_t + D x_t; head h uses group h // (H / G)."""
    T, H, P = x.shape
    share = H // B.shape[1]
    y = np.zeros((T, H, P))
    for h in range(H):
        S = np.zeros((B.shape[2], P))
        for t in range(T):
            S = np.exp(-np.exp(a_log[h]) * dt[t, h]) * S + dt[t, h] * np.outer(B[t, h // share], x[t, h])
            y[t, h] = S.T @ C[t, h // share] + D[h] * x[t, h]
    return y


def mamba2(h, W, p, m, eps):
    T = len(h)
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, u, dt = np.split(h @ W[p + "in"].T, [inner, 2 * inner + 2 * G * N], axis=1)
    x, B, C = np.split(silu(causal_filter(u, W[p + "conv"], W[p + "conv.b"])), [inner, inner + G * N], axis=1)
    y = state_space(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + W[p + "dt_bias"]), W[p + "A_log"],
                    W[p + "D"]).reshape(T, inner)
    parts = (y * silu(z)).reshape(T, m["norm_groups"], -1)
    return (unit_rms(parts, eps).reshape(T, inner) * W[p + "norm"]) @ W[p + "o"].T


def constant_decay_memory(q, k, v, decay):
    """q, k [T, H, d], v [T, H, e], decay [H]: S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t."""
    T, H, d = q.shape
    o = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        S = np.zeros((d, v.shape[2]))
        for t in range(T):
            S = decay[h] * S + np.outer(k[t, h], v[t, h])
            o[t, h] = S.T @ q[t, h]
    return o


def lightning(h, W, p, m, eps):
    T, H = len(h), m["heads"]
    q, k, v = (silu(h @ W[p + n].T).reshape(T, H, -1) for n in "qkv")
    o = constant_decay_memory(q, k, v, m["decay"]).reshape(T, -1)
    return (unit_rms(o, eps) * W[p + "norm"] * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def temperature(p, coef, every):
    return 1.0 + coef * np.log(np.floor((p + 1) / every) + 1.0)


def slopes(heads):
    return np.array([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)])


def biased_attention(q, k, v, scale, slope=None, window=None):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]: softmax over the keys j with 0 <= i - j < window of
    scale q_i.k_j - slope_h (i - j)."""
    T, H, _ = q.shape
    share = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        lo = 0 if window is None else max(0, i - window + 1)
        dist = i - np.arange(lo, i + 1)
        for h in range(H):
            s = scale * (k[lo:i + 1, h // share] @ q[i, h]) - (0.0 if slope is None else slope[h] * dist)
            w = np.exp(s - s.max())
            out[i, h] = (w / w.sum()) @ v[lo:i + 1, h // share]
    return out


def mix_values(v, first, lam):
    return (1.0 - lam) * v + lam * first


def attention(h, W, p, m, eps, first):
    """Returns (output, the layer's own values before any mixing); ``first``: the values mixed in, or None."""
    T, H, G, d = len(h), m["heads"], m["kv_heads"], m["dim"]
    q = unit_rms((h @ W[p + "q"].T).reshape(T, H, d), eps) * W[p + "q.norm"]
    k = unit_rms((h @ W[p + "k"].T).reshape(T, G, d), eps) * W[p + "k.norm"]
    own = h @ W[p + "v"].T
    v = own if first is None else mix_values(own, first, float(W[p + "vmix"]))
    qt = m.get("q_temp")
    if qt:
        q = q * temperature(np.arange(T), qt["coef"], qt["every"])[:, None, None]
    o = biased_attention(q, k, v.reshape(T, G, -1), m["scale"], slopes(H), (m.get("mask") or {}).get("size"))
    return o.reshape(T, -1) @ W[p + "o"].T, own


def dense_ff(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def expert_ff(h, W, p):
    return np.maximum(h @ W[p + "up"].T, 0.0) ** 2 @ W[p + "down"].T


def route(h, w_router, correction, top, scale, count=1, keep=1):
    """Chosen experts [T, top] and their weights [T, top]."""
    s = sigmoid(h @ w_router.T)
    choice = s + correction
    T, X = s.shape
    size = X // count
    best_two = np.sort(choice.reshape(T, count, size), axis=2)[:, :, -2:].sum(2)
    idx, wts = np.zeros((T, top), dtype=np.int64), np.zeros((T, top))
    for t in range(T):
        allowed = np.full(X, -np.inf)
        for g in np.argsort(-best_two[t], kind="stable")[:keep]:
            allowed[g * size:(g + 1) * size] = choice[t, g * size:(g + 1) * size]
        idx[t] = np.argsort(-allowed, kind="stable")[:top]
        c = s[t, idx[t]]
        wts[t] = c / (c.sum() + 1e-20) * scale
    return idx, wts


def moe_ff(h, W, p, f):
    r = f["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    idx, wts = route(h, W[p + "router"], W[p + "correction"], r["top"], r["scale"], g["count"], g["keep"])
    out = np.zeros_like(h)
    for t in range(len(h)):
        for e, w in zip(idx[t], wts[t]):
            out[t] += w * expert_ff(h[t], W, f"{p}e{e}.")
    if f.get("shared"):
        out += expert_ff(h, W, p + "shared.")
    return out


def forward(cfg, W, tokens, return_layers=False):
    """Logits [T, vocab] of one sequence (and the stream after every layer, [L, T, width])."""
    W = {k: np.asarray(v, dtype=np.float64) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    first, streams = None, []
    for i, lc in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lc["mixer"]
        h = layer_norm(x, W[p + "norm1"], W[p + "norm1.b"], eps)
        if lc["type"] == "mamba2":
            x = x + mamba2(h, W, p + "mix.", m, eps)
        elif lc["type"] == "lightning":
            x = x + lightning(h, W, p + "mix.", m, eps)
        elif lc["type"] == "attention":
            mixes = bool(m.get("v_mix"))
            y, own = attention(h, W, p + "mix.", m, eps, first if mixes else None)
            if mixes and first is None:
                first = own
            x = x + y
        else:
            raise ValueError(lc["type"])
        f = lc.get("mlp")
        if f is not None:
            h = layer_norm(x, W[p + "norm2"], W[p + "norm2.b"], eps)
            x = x + (dense_ff(h, W, p + "mlp.") if f["kind"] == "dense" else moe_ff(h, W, p + "mlp.", f))
        streams.append(x)
    logits = layer_norm(x, W["final.norm"], W["final.norm.b"], eps) @ W["head"].T
    return (logits, np.stack(streams)) if return_layers else logits
