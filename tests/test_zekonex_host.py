"""Host-side parts of the Zekonex family (no GPU): configuration from a file's dictionary and from tensor shapes, what is
refused, the order of layer runs and the memory each of them has, stacked projections, oracle identities, kernel lists."""
import importlib.util
from pathlib import Path

import numpy as np
import pytest

from oracle import zekonex as O
from tests.util_zekonex import attn, case_mixed, case_odd, case_ones, case_wide, delta, ff, latent, model_cfg

ROOT = Path(__file__).resolve().parent.parent


def need_package():
    """The package's modules load the kernels' library when imported; where it is not built these tests are skipped."""
    pytest.importorskip("torch")
    try:
        import lit_llama._native  # noqa: F401
    except ImportError as e:
        pytest.skip(str(e))


def test_configuration_from_file():
    need_package()
    from lit_llama.zekonex import ZekonexConfig

    cfg, _ = case_mixed()
    c = ZekonexConfig.from_dict(cfg)
    assert [l.kind for l in c.layers] == ["delta", "latent_attention", "attention", "delta", "attention", "latent_attention"]
    assert (c.embed_scale, c.eps, c.residual_mult, c.vocab_size, c.n_layer) == (2.5, 1e-4, 0.35, 53, 6)
    d, l, a = c.layers[0].mixer, c.layers[1].mixer, c.layers[2].mixer
    assert (d.heads, d.kv_heads, d.dim, d.vdim, d.taps, d.unit_eps) == (6, 2, 8, 12, 3, 1e-6)
    assert (l.heads, l.nope_dim, l.rot_dim, l.v_dim, l.kv_rank, l.scale, l.gate, l.window) == (3, 10, 6, 14, 24, 0.3, "none", None)
    assert (l.rotary.dims, l.rotary.base, l.rot_layout, l.exact_weights) == (6, 300.0, "interleaved", True)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.rotary.dims, a.rotary.base) == (6, 3, 12, 10, 8, 1000.0)
    assert (a.fixed_sink, a.sink, a.gate, a.rot_layout, a.reach) == (0.0, False, False, "interleaved", None)
    assert c.layers[4].mixer.scale == 0.4 and c.layers[2].ff is None and (c.layers[1].ff, c.layers[1].limit) == (36, 0.75)
    assert ZekonexConfig.from_dict(case_ones()[0]).layers[3].mixer.rotary.dims == 0
    assert ZekonexConfig.from_dict(case_wide()[0]).loop is None


def test_configuration_from_shapes():
    need_package()
    from lit_llama.zekonex import ZekonexConfig

    cfg, W = case_mixed()
    lean = {k: v for k, v in cfg.items() if k not in ("vocab", "width")}
    lean["loop"] = {k: v for k, v in cfg["loop"].items() if k != "times"}
    lean["layers"] = []
    for lc in cfg["layers"]:
        drop = {"attention": ("heads", "kv_heads", "vdim"), "delta": ("heads", "dim", "vdim", "conv"),
                "latent_attention": ("heads", "vdim", "kv_rank")}[lc["type"]]
        m = {k: v for k, v in lc["mixer"].items() if k not in drop}
        lean["layers"].append(dict(lc, mixer=m, mlp=lc["mlp"] and {k: v for k, v in lc["mlp"].items() if k != "ff"}))
    assert ZekonexConfig.from_dict(cfg) == ZekonexConfig.from_dict(lean, {k: v.shape for k, v in W.items()})
    with pytest.raises(KeyError):
        ZekonexConfig.from_dict(lean)


def test_configurations_that_are_refused():
    need_package()
    from lit_llama.softmax_attention import SoftmaxAttentionSpec
    from lit_llama.zekonex import ZekonexConfig

    ok = (attn(2, 2, 8, 8), ff(8))
    for layers in ([(dict(ok[0], type="other"), None)], [(ok[0], {"kind": "other"})], [(attn(3, 2, 8, 8), None)], [(delta(3, 2, 8, 8), None)],
                   [(attn(2, 2, 8, 8, rot=(5, 10.0)), None)], [(attn(2, 2, 8, 8, rot=(10, 10.0)), None)], [(latent(2, 8, 3, 8, 8), None)]):
        with pytest.raises(ValueError):
            ZekonexConfig.from_dict(model_cfg(11, 16, layers))
    for loop in ((1, 1, 2), (0, 2, 2), (-1, 1, 2), (0, 1, 0)):
        with pytest.raises(ValueError):
            ZekonexConfig.from_dict(model_cfg(11, 16, [ok], loop=loop))
    kw = dict(width=8, heads=1, kv_heads=1, dim=8, vdim=8, scale=1.0, eps=1e-5)
    for bad in (dict(sink=True, fixed_sink=0.0), dict(rot_layout="other"), dict(rot_layout="interleaved", own_values=False)):
        with pytest.raises(ValueError):
            SoftmaxAttentionSpec(**kw, **bad)


@pytest.mark.parametrize("loop,want", [
    (None, [(0, None), (1, None), (2, None)]),
    ((0, 3, 1), [(0, 0), (1, None), (2, None)]),
    ((1, 2, 3), [(0, None), (1, 0), (1, 1), (1, 2), (2, None)]),
    ((1, 3, 2), [(0, None), (1, 0), (2, None), (1, 1), (2, None)]),
    ((0, 2, 2), [(0, 0), (1, None), (0, 1), (1, None), (2, None)]),
])
def test_order_of_layer_runs(loop, want):
    need_package()
    from lit_llama.zekonex import ZekonexConfig

    cfg = model_cfg(11, 16, [(attn(2, 2, 8, 8), None), (delta(2, 2, 8, 8), None), (latent(2, 8, 2, 8, 8), None)], loop=loop)
    assert ZekonexConfig.from_dict(cfg).layer_runs() == want == O.layer_order(cfg)


def host_model(case):
    import torch
    from lit_llama.zekonex import Zekonex, ZekonexConfig

    cfg, W = case()
    m = Zekonex(ZekonexConfig.from_dict(cfg), dtype=torch.float32, device="cpu")
    m.load_tensors(lambda n: torch.from_numpy(np.asarray(W[n])).to(torch.bfloat16))
    return cfg, W, m


def test_every_run_of_a_layer_has_its_own_memory():
    need_package()
    cfg, W, m = host_model(case_mixed)
    assert [(r.block.index, r.step) for r in m.runs] == O.layer_order(cfg)
    m._begin(2, 48, True)
    # delta state: runs 0 and 3, 6, 9 (layer 3 in three passes); rings: layers 1, 2 in three passes, then 4 and 5
    assert [tuple(t.shape) for t in m.states] == [(2, 2, 2 * 16 + 72), (2, 6, 8, 12)] + 3 * [(2, 4, 2 * 40 + 24), (2, 4, 10, 6)]
    loop_caches = [(2, 48, 30), (2, 48, 36), (2, 48, 30)]
    assert [tuple(t.shape) for t in m.kv_caches] == 3 * loop_caches + [(2, 48, 20), (2, 48, 8), (2, 48, 14)]
    assert len({t.data_ptr() for t in m.states + m.kv_caches}) == len(m.states) + len(m.kv_caches)
    used = [(r.cache_at, len(r.block.mix.cache_shapes(1, 1))) for r in m.runs if r.ring >= 0]
    assert sorted(i for a, n in used for i in range(a, a + n)) == list(range(len(m.kv_caches)))
    assert sorted(i for r in m.runs for i in range(r.state_at, r.state_at + len(r.block.mix.state_shapes(1)))) == list(range(len(m.states)))
    assert m._piece(48) == 48 and m.rope_table(m.blocks[1].mix.spec.rotary).shape == (1024, 3, 2)


@pytest.mark.parametrize("case", [case_mixed, case_odd, case_ones])
def test_stacked_projections_hold_every_tensor_once(case):
    """The input projection's rows are [mixer; gate; up] with zeros between, the output projection's columns [W_o | W_down]; queries
    and keys of rotated heads are stored even dimensions first on both sides."""
    need_package()
    cfg, W, m = host_model(case)
    for b, lc in zip(m.blocks, cfg["layers"]):
        p, f = f"l{b.index}.", lc.get("mlp")
        w_in, w_out = b.w_in.numpy(), b.w_out.numpy()
        names = {"attention": "qkv", "delta": "qkvgab", "latent_attention": ("q", "dkv")}[lc["type"]]
        total = sum(np.abs(W[p + "mix." + n]).sum() for n in names) + (np.abs(W[p + "mlp.gate"]).sum() + np.abs(W[p + "mlp.up"]).sum() if f else 0)
        assert np.abs(w_in).sum() == pytest.approx(total, rel=1e-5)
        assert np.array_equal(w_out[:, :b.mix.out_cols], W[p + "mix.o"].astype(np.float32))
        if f:
            assert np.array_equal(w_in[b.ff_in:b.ff_in + f["ff"]], W[p + "mlp.gate"].astype(np.float32)) and b.ff_in % 8 == 0 == b.ff_out % 8
            assert np.array_equal(w_out[:, b.ff_out:b.ff_out + f["ff"]], W[p + "mlp.down"].astype(np.float32))
            assert np.array_equal(b.mlp.bias.numpy(), np.concatenate([W[p + "mlp.gate.b"], W[p + "mlp.up.b"]]).astype(np.float32))
        if lc["type"] == "attention" and (lc["mixer"].get("rot") or {}).get("dims"):
            d, r = lc["mixer"]["dim"], lc["mixer"]["rot"]["dims"]
            order = list(range(0, r, 2)) + list(range(1, r, 2)) + list(range(r, d))
            for n in "qk":
                w = W[p + "mix." + n].reshape(-1, d, cfg["width"])[:, order].reshape(-1, cfg["width"])
                assert np.array_equal(w_in[b.mix.cols[n]:b.mix.cols[n] + len(w)], w.astype(np.float32))
            assert np.array_equal(b.mix.sink.numpy(), np.zeros(lc["mixer"]["heads"]))


def test_interleaved_pairs_turned_as_halves():
    """Reordering heads and turning (i, i + dims/2) is turning (2i, 2i + 1) and reordering: scores are the same."""
    need_package()
    from lit_llama.rotary import RotarySpec
    from lit_llama.softmax_attention import SoftmaxAttentionSpec
    from oracle.tebodra import rotate

    r = np.random.RandomState(0)
    s = SoftmaxAttentionSpec(width=8, heads=2, kv_heads=2, dim=10, vdim=4, scale=1.0, eps=1e-5, rotary=RotarySpec(6, 100.0), rot_layout="interleaved")
    order = s.head_order().numpy()
    x, p = r.randn(5, 2, 10), np.arange(40, 45)
    assert np.allclose(rotate(x[..., order], {"base": 100.0, "dims": 6}, p), O.turn(x, p, 6, 100.0)[..., order])


def test_family_kernel_list():
    spec = importlib.util.spec_from_file_location("llb200_build", ROOT / "lit-llama-ja_b200" / "build.py")
    build = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(build)
    assert {"delta_rule", "delta_chunk", "rotary_attn", "latent_attn", "short_conv"} <= set(build.FAMILY_SOURCES["Zekonex"])
    need_package()
    from lit_llama.registry import architectures

    assert "Zekonex" in architectures()


def test_oracle_identities():
    r = np.random.RandomState(0)
    # one more unit in the denominator is a key of score 0 without value
    q, k, v = r.randn(9, 4, 6), r.randn(9, 2, 6), r.randn(9, 2, 5)
    a, plain = O.causal_softmax(q, k, v, 0.7, 1.0), O.causal_softmax(q, k, v, 0.7, 0.0)
    s = 0.7 * k[:4, 1] @ q[3, 2]
    assert np.allclose(a[3, 2], (np.exp(s) / (1 + np.exp(s).sum())) @ v[:4, 1]) and np.allclose(plain[0], v[0][[0, 0, 1, 1]])
    # a turn keeps lengths, and dot products depend on the distance alone
    x, y = r.randn(1, 1, 8), r.randn(1, 1, 8)
    dots = [np.sum(O.turn(x, [p], 8, 50.0) * O.turn(y, [p - 7], 8, 50.0)) for p in (7, 100, 4000)]
    assert np.allclose(dots, dots[0]) and np.allclose(O.turn(x, [9], 4, 50.0)[..., 4:], x[..., 4:])
    # a memory without fading and with full strength returns the last value written under each of its orthogonal keys
    n = 5
    keys = np.eye(n)[r.randint(n, size=30)][:, None]
    val = r.randn(30, 1, 3)
    o, S = O.delta_memory(keys, keys, val, np.ones((30, 1)), np.ones((30, 1)))
    assert np.allclose(o, val)
    for i in range(n):
        last = np.flatnonzero(keys[:, 0, i])
        assert np.allclose(S[0][i], val[last[-1], 0] if len(last) else 0.0)
    # in two halves
    g, b = r.uniform(0.5, 1, (30, 2)), r.uniform(0, 1, (30, 2))
    q, k, v = r.randn(30, 1, 4), O.unit_vector(r.randn(30, 1, 4)), r.randn(30, 2, 3)
    whole, S = O.delta_memory(q, k, v, g, b)
    first, mid = O.delta_memory(q[:13], k[:13], v[:13], g[:13], b[:13])
    second, end = O.delta_memory(q[13:], k[13:], v[13:], g[13:], b[13:], mid)
    assert np.allclose(np.concatenate([first, second]), whole) and np.allclose(end, S)
    assert np.allclose(O.clamped_unit(np.array([9.0, -9.0]), np.array([9.0, -9.0]), 2.0),
                       [2 * 3 / (1 + np.exp(-3.404)), 9 / (1 + np.exp(9 * 1.702))])
