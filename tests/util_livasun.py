"""Builders shared by the Livasun tests: small random models written as model folders (config.json + safetensors) and
loaded back through the package's registry, and comparisons against the float64 oracle (oracle/livasun.py)."""
import json

import numpy as np
import torch

from tests.util_bededra import agrees, bf16, load, rel_err, run_schedule      # noqa: F401  (model-agnostic helpers)

TOL32 = 2e-4


def mamba(heads, vdim, state, groups=1, norm_groups=1, conv=4):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups,
                                        "conv": conv}}


def lightning(decay, dim, vdim):
    return {"type": "lightning", "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}}


def attn(heads, kv_heads, dim, vdim, window, v_mix=True, temp=(0.4, 6), scale=None):
    """``window`` None: every earlier token is visible; ``temp`` None: no query temperature."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
         "v_mix": v_mix}
    if window is not None:
        m["mask"] = {"size": window}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None, count=1, keep=1, scale=1.5):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if count > 1:
        f["router"]["groups"] = {"count": count, "keep": keep}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def model_cfg(vocab, width, layers, eps=1e-5, scale=3.0):
    """``layers``: (mixer entry from mamba() / lightning() / attn(), feed-forward entry or None)."""
    return {"architecture": "Livasun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": [dict(m, mlp=f) for m, f in layers]}


def random_weights(cfg, seed=0, qk_gain=1.5):
    """Every tensor of the design with values that keep activations of order one; already rounded to bfloat16."""
    r = np.random.RandomState(seed)
    E, W = cfg["width"], {}

    def lin(o, i, gain=1.0):
        return r.randn(o, i) * gain / np.sqrt(i)

    def norm(name, n):
        W[name], W[name + ".b"] = 1 + 0.2 * r.randn(n), 0.3 * r.randn(n)

    W["embed"] = r.randn(cfg["vocab"], E)
    W["head"] = lin(cfg["vocab"], E)
    norm("final.norm", E)
    for i, lc in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lc["mixer"]
        norm(p + "norm1", E)
        H = m["heads"]
        if lc["type"] == "mamba2":
            inner, gn = H * m["vdim"], m["groups"] * m["state"]
            W[p + "mix.in"] = lin(2 * inner + 2 * gn + H, E, 1.3)
            W[p + "mix.conv"], W[p + "mix.conv.b"] = 0.6 * r.randn(inner + 2 * gn, m["conv"]), 0.2 * r.randn(inner + 2 * gn)
            W[p + "mix.dt_bias"], W[p + "mix.A_log"], W[p + "mix.D"] = r.uniform(-3, 0.5, H), r.uniform(-2, 1, H), r.randn(H)
            W[p + "mix.norm"], W[p + "mix.o"] = 1 + 0.1 * r.randn(inner), lin(E, inner)
        elif lc["type"] == "lightning":
            D, V = m["dim"], m["vdim"]
            W[p + "mix.q"], W[p + "mix.k"], W[p + "mix.v"] = lin(H * D, E, 1.5), lin(H * D, E, 1.5), lin(H * V, E, 1.5)
            W[p + "mix.g"], W[p + "mix.o"], W[p + "mix.norm"] = lin(H * V, E), lin(E, H * V), 1 + 0.1 * r.randn(H * V)
        else:
            G, D, V = m["kv_heads"], m["dim"], m["vdim"]
            W[p + "mix.q"], W[p + "mix.k"], W[p + "mix.v"] = lin(H * D, E), lin(G * D, E), lin(G * V, E)
            W[p + "mix.q.norm"], W[p + "mix.k.norm"] = qk_gain * (1 + 0.2 * r.randn(D)), 1 + 0.2 * r.randn(D)
            W[p + "mix.vmix"] = np.array(r.uniform(0.2, 0.8))
            W[p + "mix.o"] = lin(E, H * V)
        f = lc.get("mlp")
        if f is None:
            continue
        norm(p + "norm2", E)
        if f["kind"] == "dense":
            W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"] = lin(f["ff"], E), lin(f["ff"], E), lin(E, f["ff"])
        else:
            X = f["router"]["experts"]
            W[p + "mlp.router"], W[p + "mlp.correction"] = lin(X, E, 2.0), r.uniform(-1.2, 0.2, X)     # choice scores of both signs
            for q, ff in [(f"e{e}.", f["expert"]["ff"]) for e in range(X)] + ([("shared.", f["shared"]["ff"])] if f.get("shared") else []):
                W[p + "mlp." + q + "up"], W[p + "mlp." + q + "down"] = lin(ff, E), lin(E, ff)
    return {k: bf16(v) for k, v in W.items()}


def case_mixed(seed=0):
    """Sizes that share nothing with each other, the mixers in an order of its own, every kind of feed-forward and none, an
    attention layer that mixes no values between two that do."""
    layers = [
        (attn(6, 2, 8, 12, window=7, temp=(0.5, 5)), moe(6, 2, 12, shared=20, count=3, keep=2, scale=1.7)),
        (mamba(3, 8, 10, norm_groups=3, conv=3), dense(24)),
        (attn(2, 1, 16, 4, window=9, v_mix=False, temp=(0.3, 16)), None),
        (lightning([0.6, 0.97], 6, 10), moe(8, 3, 10, count=2, keep=1, scale=0.8)),
        (attn(4, 4, 12, 6, window=11, temp=(0.2, 3), scale=0.4), dense(40)),
        (mamba(4, 6, 20, groups=2, norm_groups=1, conv=2), None),
        (lightning([0.9, 0.5, 0.999], 12, 4), moe(4, 2, 16, shared=8)),
    ]
    cfg = model_cfg(53, 40, layers, eps=1e-4, scale=2.5)
    return cfg, random_weights(cfg, seed)


def case_ones(seed=1):
    """Sizes that are 1 or equal where a real model's differ: one head, one tap, one expert, groups of one expert, a window of
    one position, a window longer than any test sequence, no temperature, decays of zero and one."""
    layers = [
        (attn(1, 1, 8, 8, window=1, temp=(0.5, 1)), moe(1, 1, 8)),
        (mamba(1, 8, 8, conv=1), moe(4, 2, 8, shared=8, count=4, keep=2, scale=1.0)),
        (attn(2, 2, 4, 4, window=1000, temp=None), dense(8)),
        (lightning([0.0, 1.0], 1, 4), moe(4, 4, 8, count=2, keep=2)),
        (attn(2, 2, 4, 4, window=None, temp=(0.7, 1000)), None),
    ]
    cfg = model_cfg(19, 8, layers, eps=1e-6, scale=1.0)
    cfg["layers"][0]["mixer"]["v_mix"] = False        # its values have another size than the others'
    return cfg, random_weights(cfg, seed)


def case_odd(seed=2):
    """Nothing is a multiple of 4: every kernel takes its padded / unaligned path."""
    layers = [
        (attn(3, 3, 5, 7, window=6), moe(9, 2, 11, shared=7, count=3, keep=1)),
        (mamba(5, 3, 7, groups=5, norm_groups=5, conv=5), dense(13)),
        (lightning([0.8, 0.95, 0.7], 9, 11), None),
        (attn(3, 3, 11, 7, window=9, temp=(0.1, 2)), dense(9)),
    ]
    cfg = model_cfg(37, 30, layers, eps=1e-6)
    return cfg, random_weights(cfg, seed)


def case_wide(seed=3):
    """Head sizes in multiples of 8 (the tensor-core form in bf16), different key and value sizes, prompts longer than a
    query tile with window edges inside tiles, long parts in the gated norms."""
    layers = [
        (attn(4, 2, 32, 16, window=40, temp=(0.3, 20)), moe(8, 2, 24, shared=40, count=4, keep=2)),
        (mamba(8, 40, 16, groups=2), None),
        (attn(4, 1, 72, 32, window=23, scale=0.1), dense(48)),
        (lightning([0.9, 0.99, 0.999], 24, 96), None),
    ]
    cfg = model_cfg(83, 64, layers, eps=1e-5)
    return cfg, random_weights(cfg, seed)


def case_one_kind(kind, seed=4):
    """Models with a single kind of mixer: recurrent state without rings, or rings without recurrent state."""
    layers = {"mamba2": [(mamba(2, 8, 12, groups=2, norm_groups=2), dense(20)), (mamba(4, 4, 6), None)],
              "lightning": [(lightning([0.9], 8, 8), dense(20)), (lightning([0.5, 0.99], 4, 12), None)],
              "attention": [(attn(2, 2, 16, 16, window=9), dense(16)), (attn(4, 2, 8, 16, window=5), None)]}[kind]
    cfg = model_cfg(29, 24, layers)
    return cfg, random_weights(cfg, seed)


def write_model(folder, cfg, W):
    from lit_llama.safetensors_io import save_safetensors

    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    save_safetensors({k: torch.from_numpy(np.asarray(v, dtype=np.float32)).to(torch.bfloat16) for k, v in W.items()},
                     folder / "model.safetensors")
    return folder
