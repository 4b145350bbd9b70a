"""Plain, slow float64 statement of the Zekonex design, one function per mechanism (numpy only; test infrastructure, never
imported by the product).  It works on a whole sequence at once and keeps no cache: whatever schedule the product runs
(portions, single tokens, rings, recurrent state handed from step to step), its logits must equal these.

The stream starts as ``embed[token] * s_e``.  A layer has one norm whose output both of its sublayers read:

    h = rmsnorm(x) * w;      x <- x + r * ( mixer(h) + ff(h) )            (ff may be absent)

A range of layers may run several times in a row with the same weights; right before its pass t the learned vector
``loop.step[t]`` joins the stream.  Mixers: ``attention`` (softmax with one more unit in the denominator, neighbouring
dimensions turned in pairs), ``delta`` (a matrix memory written by a gated delta rule) and ``latent_attention`` (keys and
values expanded from one low-rank row per token).  Feed-forward: a gated unit with clamped inputs and biases.
Logits: head . (rmsnorm(x) * w_f).

Checkpoint names: ``embed``, ``head``, ``final.norm``, ``loop.step``; per layer i ``l<i>.norm1``, ``l<i>.mix.*``,
``l<i>.mlp.*``; Linear weights are [out, in].
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


def unit_vector(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def turn(x, pos, dims, base):
    """x [T, heads, d]: of every head's first ``dims`` numbers, (2i, 2i + 1) turn together by pos * base^(-2i / dims)."""
    out = np.array(x, dtype=np.float64)
    for i in range(dims // 2):
        a = np.asarray(pos, dtype=np.float64)[:, None] * base ** (-2.0 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)
    return out


def causal_softmax(q, k, v, scale, extra):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]: weights exp(s_j) / (extra + sum exp(s_j)) over the keys j <= i."""
    T, H, _ = q.shape
    share = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        for h in range(H):
            s = scale * (k[:i + 1, h // share] @ q[i, h])
            top = max(s.max(), 0.0) if extra else s.max()
            w = np.exp(s - top)
            out[i, h] = (w / (w.sum() + extra * np.exp(-top))) @ v[:i + 1, h // share]
    return out


def attention(h, W, p, m, pos):
    T = len(h)
    q, k, v = (h @ W[p + n].T for n in "qkv")
    q, k, v = q.reshape(T, m["heads"], -1), k.reshape(T, m["kv_heads"], -1), v.reshape(T, m["kv_heads"], -1)
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    q, k = (turn(t, pos, rot["dims"], rot["base"]) for t in (q, k))
    return causal_softmax(q, k, v, m["scale"], 1.0).reshape(T, -1) @ W[p + "o"].T


def causal_filter(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), nothing before the first token."""
    taps = w.shape[1]
    past = np.concatenate([np.zeros((taps - 1, u.shape[1])), u])
    return sum(past[j:j + len(u)] * w[:, j] for j in range(taps))


def delta_memory(q, k, v, g, beta, S=None):
    """q, k [T, G, n], v [T, H, e], g and beta [T, H]; head h uses q/k head h // (H / G).  Per token: the memory fades by g, what it
    returns for k is compared with v, beta of the difference is written under k, then q reads.  Returns (o [T, H, e], S)."""
    T, H, e = v.shape
    share = H // k.shape[1]
    S = np.zeros((H, k.shape[2], e)) if S is None else np.array(S, dtype=np.float64)
    o = np.zeros((T, H, e))
    for h in range(H):
        for t in range(T):
            kt, qt = k[t, h // share], q[t, h // share]
            S[h] *= g[t, h]
            S[h] += np.outer(kt, beta[t, h] * (v[t, h] - S[h].T @ kt))
            o[t, h] = S[h].T @ qt
    return o, S


def delta_gates(a, b, dt_bias, a_log):
    """(decay, write strength) of the projections a and b [T, H]."""
    return np.exp(-np.exp(a_log) * softplus(a + dt_bias)), sigmoid(b)


def delta(h, W, p, m, eps):
    T, H, G, n, e = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_filter(h @ W[p + s].T, W[p + s + ".conv"])) for s in "qkv")
    q, k = unit_vector(q.reshape(T, G, n)) * n ** -0.5, unit_vector(k.reshape(T, G, n))
    g, beta = delta_gates(h @ W[p + "a"].T, h @ W[p + "b"].T, W[p + "dt_bias"], W[p + "A_log"])
    o, _ = delta_memory(q, k, v.reshape(T, H, e), g, beta)
    o = unit_rms(o, eps) * W[p + "norm"] * silu(h @ W[p + "g"].T).reshape(T, H, e)
    return o.reshape(T, H * e) @ W[p + "o"].T


def latent_attention(h, W, p, m, eps, pos):
    T, H, n, r, R = len(h), m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    q = (h @ W[p + "q"].T).reshape(T, H, n + r)
    d = h @ W[p + "dkv"].T
    c = unit_rms(d[:, :R], eps) * W[p + "dkv.norm"]
    k_rot = turn(d[:, None, R:], pos, rot["dims"], rot["base"])
    q = np.concatenate([q[..., :n], turn(q[..., n:], pos, rot["dims"], rot["base"])], axis=-1)
    k = np.concatenate([(c @ W[p + "uk"].T).reshape(T, H, n), np.repeat(k_rot, H, axis=1)], axis=-1)
    v = (c @ W[p + "uv"].T).reshape(T, H, -1)
    return causal_softmax(q, k, v, m["scale"], 0.0).reshape(T, -1) @ W[p + "o"].T


def clamped_unit(g, u, limit):
    g, u = np.minimum(g, limit), np.clip(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def dense_ff(h, W, p, limit):
    g, u = (h @ W[p + n].T + W[p + n + ".b"] for n in ("gate", "up"))
    return clamped_unit(g, u, limit) @ W[p + "down"].T + W[p + "down.b"]


def layer_order(cfg):
    """(layer, pass it opens or None) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return [(i, None) for i in range(a)] + [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)] \
        + [(i, None) for i in range(b, n)]


def forward(cfg, W, tokens, return_layers=False):
    """float64 logits [T, vocab] of one sequence; optionally the stream after every layer run."""
    eps, r = cfg["norm"]["eps"], cfg["residual_mult"]
    pos = np.arange(len(tokens))
    x = W["embed"][np.asarray(tokens)] * (cfg.get("embedding") or {}).get("scale", 1.0)
    streams = []
    for i, step in layer_order(cfg):
        lc, p = cfg["layers"][i], f"l{i}."
        if step is not None:
            x = x + W["loop.step"][step]
        h = unit_rms(x, eps) * W[p + "norm1"]
        if lc["type"] == "attention":
            y = attention(h, W, p + "mix.", lc["mixer"], pos)
        elif lc["type"] == "delta":
            y = delta(h, W, p + "mix.", lc["mixer"], eps)
        else:
            y = latent_attention(h, W, p + "mix.", lc["mixer"], eps, pos)
        if lc.get("mlp"):
            y = y + dense_ff(h, W, p + "mlp.", lc["mlp"]["limit"])
        x = x + r * y
        streams.append(x)
    logits = (unit_rms(x, eps) * W["final.norm"]) @ W["head"].T
    return (logits, streams) if return_layers else logits
