"""Builders shared by the Zekonex tests: small random models written as model folders (config.json + safetensors) and loaded
back through the package's registry, and comparisons against the float64 oracle (oracle/zekonex.py)."""
import numpy as np
import torch

from tests.util_bededra import bf16, load, rel_err, run_schedule      # noqa: F401  (model-agnostic helpers)
from tests.util_livasun import write_model                            # noqa: F401

TOL32 = 2e-4


def agrees(got, want, dtype):
    """fp32: summation order only.  bf16: operands are rounded in every layer; nothing is chosen, so no token may be far off."""
    if dtype == torch.float32:
        return rel_err(got, want) < TOL32
    per_token = np.abs(got - want).reshape(-1, got.shape[-1]).max(-1) / np.abs(want).max()
    return bool(np.median(per_token) < 0.03 and per_token.max() < 0.12)


def attn(heads, kv_heads, dim, vdim, rot=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "attention", "mixer": m}


def delta(heads, kv_heads, dim, vdim, conv=4):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def latent(heads, dim, rot_dim, vdim, rank, base=500.0, scale=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "rot": {"dims": rot_dim, "base": base},
                      "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}}


def ff(inner, limit=2.0):
    return {"kind": "dense", "ff": inner, "limit": limit}


def model_cfg(vocab, width, layers, eps=1e-5, scale=3.0, r=0.4, loop=None):
    """``layers``: (mixer entry from attn() / delta() / latent(), feed-forward entry or None); ``loop``: (start, stop, times)."""
    cfg = {"architecture": "Zekonex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
           "residual_mult": r, "layers": [dict(m, mlp=f) for m, f in layers]}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def random_weights(cfg, seed=0, qk_gain=1.5):
    """Every tensor of the design with values that keep activations of order one; already rounded to bfloat16."""
    g = np.random.RandomState(seed)
    E, W = cfg["width"], {}

    def lin(o, i, gain=1.0):
        return g.randn(o, i) * gain / np.sqrt(i)

    W["embed"], W["head"], W["final.norm"] = g.randn(cfg["vocab"], E), lin(cfg["vocab"], E), 1 + 0.2 * g.randn(E)
    if cfg.get("loop"):
        W["loop.step"] = g.randn(cfg["loop"]["times"], E)
    for i, lc in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", lc["mixer"]
        W[f"l{i}.norm1"] = 1 + 0.2 * g.randn(E)
        H, D, V = m["heads"], m["dim"], m["vdim"]
        if lc["type"] == "attention":
            G = m["kv_heads"]
            W[p + "q"], W[p + "k"], W[p + "v"], W[p + "o"] = lin(H * D, E, qk_gain), lin(G * D, E, qk_gain), lin(G * V, E), lin(E, H * V)
        elif lc["type"] == "delta":
            G = m["kv_heads"]
            for s, n in (("q", G * D), ("k", G * D), ("v", H * V)):
                W[p + s], W[p + s + ".conv"] = lin(n, E, 1.5), 0.6 * g.randn(n, m["conv"])
            W[p + "a"], W[p + "b"], W[p + "g"] = lin(H, E), lin(H, E, 2.0), lin(H * V, E)
            W[p + "A_log"], W[p + "dt_bias"] = g.uniform(-3, 1, H), g.uniform(-3, 0.5, H)
            W[p + "norm"], W[p + "o"] = 1 + 0.2 * g.randn(V), lin(E, H * V)
        else:
            r, R = m["rot_dim"], m["kv_rank"]
            W[p + "q"], W[p + "dkv"], W[p + "dkv.norm"] = lin(H * (D + r), E, qk_gain), lin(R + r, E), 1 + 0.2 * g.randn(R)
            W[p + "uk"], W[p + "uv"], W[p + "o"] = lin(H * D, R, qk_gain), lin(H * V, R), lin(E, H * V)
        if lc.get("mlp"):
            F, q = lc["mlp"]["ff"], f"l{i}.mlp."
            W[q + "gate"], W[q + "up"], W[q + "down"] = lin(F, E, 1.5), lin(F, E, 1.5), lin(E, F)
            W[q + "gate.b"], W[q + "up.b"], W[q + "down.b"] = 0.5 * g.randn(F), 0.5 * g.randn(F), 0.3 * g.randn(E)
    return {k: bf16(v) for k, v in W.items()}


def case_mixed(seed=0):
    """Sizes that share nothing with each other, the mixers in an order of its own, a loop of three passes over layers that start
    with one kind and end with another, a layer without feed-forward inside it and one outside."""
    layers = [
        (delta(6, 2, 8, 12, conv=3), ff(20, 1.25)),
        (latent(3, 10, 6, 14, 24, base=300.0, scale=0.3), ff(36, 0.75)),
        (attn(6, 3, 12, 10, rot=(8, 1000.0)), None),
        (delta(4, 4, 10, 6, conv=5), ff(28, 3.0)),
        (attn(4, 1, 20, 8, rot=(20, 50.0), scale=0.4), ff(12, 1.0)),
        (latent(5, 4, 2, 8, 12), None),
    ]
    cfg = model_cfg(53, 40, layers, eps=1e-4, scale=2.5, r=0.35, loop=(1, 4, 3))
    return cfg, random_weights(cfg, seed)


def case_ones(seed=1):
    """Sizes that are 1 or equal where a real model's differ: one head, one tap, one turning pair, one unit, a loop over every layer
    that runs once, a multiplier of one."""
    layers = [
        (attn(1, 1, 8, 8, rot=(2, 10.0)), ff(1, 0.5)),
        (delta(1, 1, 8, 8, conv=1), ff(8)),
        (latent(1, 8, 2, 8, 8), None),
        (attn(2, 2, 4, 4), ff(8)),
        (delta(2, 2, 1, 1, conv=2), None),
    ]
    cfg = model_cfg(19, 8, layers, eps=1e-6, scale=1.0, r=1.0, loop=(0, 5, 1))
    return cfg, random_weights(cfg, seed)


def case_odd(seed=2):
    """Nothing is a multiple of 4: every kernel takes its padded / unaligned path.  The loop ends with the model's last layer."""
    layers = [
        (attn(3, 3, 6, 7, rot=(2, 30.0)), ff(11)),
        (delta(5, 5, 3, 7, conv=6), ff(13, 1.0)),
        (latent(3, 5, 6, 7, 9), ff(9)),
    ]
    cfg = model_cfg(37, 30, layers, eps=1e-6, r=0.5, loop=(2, 3, 2))
    return cfg, random_weights(cfg, seed)


def case_wide(seed=3):
    """Head sizes in multiples of 8 (the tensor-core forms in bf16), different key and value sizes, prompts of several chunks and
    longer than a query tile; no loop."""
    layers = [
        (attn(4, 2, 32, 16, rot=(24, 1e4)), ff(48)),
        (delta(6, 3, 24, 40), ff(40, 1.5)),
        (latent(4, 24, 8, 16, 40), ff(56)),
        (delta(2, 1, 72, 16, conv=3), None),
        (attn(4, 1, 72, 40, rot=(72, 100.0), scale=0.1), None),
    ]
    cfg = model_cfg(83, 64, layers, eps=1e-5)
    return cfg, random_weights(cfg, seed)


def case_one_kind(kind, seed=4):
    """Models with a single kind of mixer: recurrent state without rings, or rings without recurrent state."""
    layers = {"delta": [(delta(4, 2, 8, 12), ff(20)), (delta(2, 2, 6, 6, conv=2), None)],
              "attention": [(attn(2, 2, 16, 16, rot=(16, 100.0)), ff(16)), (attn(4, 2, 8, 16), None)],
              "latent_attention": [(latent(2, 8, 4, 8, 16), ff(16)), (latent(4, 6, 2, 10, 8), None)]}[kind]
    cfg = model_cfg(29, 24, layers, loop=(1, 2, 2))
    return cfg, random_weights(cfg, seed)
