"""Host-side parts of the Livasun family (no GPU): configuration from a file's dictionary and from tensor shapes, which layer
gives its values to the others, what is refused, ring arithmetic of sliding windows, oracle identities, kernel lists."""
import importlib.util

import numpy as np
import pytest

from oracle import livasun as O
from tests.util_livasun import attn, case_mixed, case_ones, dense, lightning, model_cfg, moe


def need_package():
    """The package's modules load the kernels' library when imported; where it is not built these tests are skipped."""
    pytest.importorskip("torch")
    try:
        import lit_llama._native  # noqa: F401
    except ImportError as e:
        pytest.skip(str(e))


def test_configuration_from_file():
    need_package()
    from lit_llama.livasun import LivasunConfig
    from lit_llama.moe import MoESpec

    cfg, _ = case_mixed()
    c = LivasunConfig.from_dict(cfg)
    assert [l.kind for l in c.layers] == ["attention", "mamba2", "attention", "lightning", "attention", "mamba2", "lightning"]
    assert (c.embed_scale, c.eps, c.values_of) == (2.5, 1e-4, 0)
    a, plain, b = c.layers[0].mixer, c.layers[2].mixer, c.layers[4].mixer
    assert (a.window, a.temp_coef, a.temp_every, a.head_norm, a.distance_bias, a.gate) == (7, 0.5, 5, True, True, False)
    assert (a.v_mix, plain.v_mix, b.v_mix) == (False, False, True)               # the first one only gives its values
    assert b.scale == 0.4 and b.reach == 11
    f = c.layers[0].mlp
    assert isinstance(f, MoESpec) and (f.experts, f.top, f.groups, f.keep_groups, f.group_top, f.weight_scale) == (6, 2, 3, 2, 2, 1.7)
    assert (f.score, f.unit, f.correction, f.router_bias, f.shared_ff, f.shared_gate) == ("sigmoid", "relu2", True, False, 20, False)
    assert c.layers[3].mlp.shared_ff is None and c.layers[2].mlp is None and c.layers[4].mlp == 40
    assert c.layers[6].mlp.groups == 1 and c.layers[3].mixer.decay == (0.6, 0.97)
    one = LivasunConfig.from_dict(case_ones()[0])
    assert one.values_of == 2 and one.layers[4].mixer.window is None and one.layers[4].mixer.reach is None
    assert one.layers[2].mixer.temp_every == 0


def test_configuration_from_shapes():
    need_package()
    from lit_llama.livasun import LivasunConfig

    cfg, W = case_mixed()
    lean = {k: v for k, v in cfg.items() if k not in ("vocab", "width")}
    lean["layers"] = []
    for lc in cfg["layers"]:
        m = {k: v for k, v in lc["mixer"].items() if k not in ("heads", "dim", "vdim", "kv_heads", "conv")}
        f = lc["mlp"] and {k: v for k, v in lc["mlp"].items() if k not in ("ff", "expert")}
        lean["layers"].append(dict(lc, mixer=m, mlp=f))
    c, c2 = LivasunConfig.from_dict(cfg), LivasunConfig.from_dict(lean, {k: v.shape for k, v in W.items()})
    assert c == c2
    with pytest.raises(KeyError):
        LivasunConfig.from_dict(lean)


def test_configurations_that_are_refused():
    need_package()
    from lit_llama.livasun import LivasunConfig

    ok = (attn(2, 2, 8, 8, window=4), dense(8))
    for layers in ([ok, (attn(2, 1, 8, 8, window=4), None)],                     # value projections of different sizes are not mixed
                   [(dict(ok[0], type="other"), None)],
                   [(ok[0], {"kind": "other"})],
                   [(attn(3, 2, 8, 8, window=4), None)],                         # 3 query heads over 2
                   [({"type": "lightning", "mixer": {"heads": 3, "dim": 4, "vdim": 4, "decay": [0.5, 0.9]}}, None)]):
        with pytest.raises(ValueError):
            LivasunConfig.from_dict(model_cfg(11, 16, layers))
    bad = LivasunConfig.from_dict(model_cfg(11, 16, [(ok[0], moe(4, 3, 8, count=2, keep=1))]))      # 3 choices out of 2 experts
    from lit_llama.moe import MoE

    import torch
    with pytest.raises(ValueError):
        MoE(bad.layers[0].mlp, torch.float32, "cpu")


def test_rings_of_sliding_windows():
    """A step never writes a slot that one of its own queries still reads."""
    need_package()
    from lit_llama.cache import max_portion, ring_length

    for window in (1, 4, 9):
        for portion in (1, 2, 8):
            ring = ring_length(1000, window, portion)
            assert max_portion(ring, 1000, window) == portion
            for first in range(0, 40):
                written = {(first + t) % ring for t in range(portion)}
                for t in range(portion):
                    reads = {j % ring for j in range(max(0, first + t - window + 1), first)}
                    assert not (reads & written)


def test_model_memory_plan_and_weight_loading_on_the_host():
    need_package()
    import torch
    from lit_llama.livasun import Livasun, LivasunConfig

    cfg, W = case_mixed()
    m = Livasun(LivasunConfig.from_dict(cfg), dtype=torch.float32, device="cpu")
    m.load_tensors(lambda n: torch.from_numpy(np.asarray(W[n])).to(torch.bfloat16))
    a = m.blocks[4].mix
    assert a.v_lambda == pytest.approx(float(W["l4.mix.vmix"])) and m.blocks[0].mix.v_lambda == 0.0
    assert np.allclose(a.slopes.numpy(), [2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8])
    assert np.array_equal(m.blocks[1].norm1.b.numpy(), W["l1.norm1.b"].astype(np.float32))
    up = m.blocks[4].mlp.w_up
    assert np.array_equal(up[:40].numpy(), W["l4.mlp.gate"].astype(np.float32)) and np.array_equal(up[40:].numpy(), W["l4.mlp.up"].astype(np.float32))
    assert m._ring_plan(64) == (64, 64, 64)
    m.prefill_portion = 3
    assert m._ring_plan(64) == (7 - 1 + 3, 9 - 1 + 3, 11 - 1 + 3)
    m._begin(2, 64, True)
    assert [tuple(t.shape) for t in m.states] == [(2, 2, 3 * 8 + 2 * 10), (2, 3, 10, 8), (2, 2, 6, 10), (2, 1, 4 * 6 + 2 * 2 * 20),
                                                  (2, 4, 20, 6), (2, 3, 12, 4)]
    assert [tuple(t.shape) for t in m.kv_caches[:2]] == [(2, 9, 16), (2, 9, 24)] and m._piece(64) == 3


def test_oracle_identities():
    r = np.random.RandomState(0)
    q, k, v = r.randn(12, 4, 6), r.randn(12, 2, 6), r.randn(12, 2, 5)
    a = O.biased_attention(q, k, v, 0.4)
    assert np.allclose(a, O.biased_attention(q, k, v, 0.4, window=12)) and not np.allclose(a, O.biased_attention(q, k, v, 0.4, window=11))
    assert np.allclose(O.biased_attention(q, k, v, 0.4, window=1), np.repeat(v, 2, axis=1))
    assert np.allclose(a, O.biased_attention(q, k, v, 0.4, slope=np.zeros(4)))
    assert np.allclose(O.slopes(8), 0.5 ** np.arange(1, 9))
    assert np.allclose(O.temperature(np.array([0, 4, 5, 8, 9]), 1.0, 5), 1 + np.log([1, 2, 2, 2, 3]))
    x = r.randn(3, 9)
    n = O.layer_norm(x, np.ones(9), np.zeros(9), 0.0)
    assert np.allclose(n.mean(1), 0) and np.allclose((n * n).mean(1), 1)
    # a decay of zero remembers nothing, a decay of one everything
    o = O.constant_decay_memory(q[:, :2], k, v, [0.0, 1.0])
    assert np.allclose(o[:, 0], (q[:, 0] * k[:, 0]).sum(1, keepdims=True) * v[:, 0])
    assert np.allclose(o[-1, 1], sum((q[-1, 1] @ k[t, 1]) * v[t, 1] for t in range(12)))
    # a correction moves the choice and not the weights; groups go by their two best
    w = np.eye(4)
    h = np.array([[1.0, 0.9, 3.0, -9.0]])
    idx, wts = O.route(h, w, np.zeros(4), 2, 2.0)
    assert sorted(idx[0]) == [0, 2] and wts.sum() == pytest.approx(2.0)
    idx, wts = O.route(h, w, np.array([0.0, 5.0, 0.0, 0.0]), 2, 1.0)
    assert sorted(idx[0]) == [1, 2] and wts[0][list(idx[0]).index(1)] == pytest.approx(O.sigmoid(0.9) / (O.sigmoid(0.9) + O.sigmoid(3.0)))
    assert sorted(O.route(h, w, np.zeros(4), 2, 1.0, 2, 1)[0][0]) == [0, 1]        # the best single expert is in the other group


def test_family_is_registered_with_its_kernels():
    need_package()
    from lit_llama.registry import architectures

    assert "Livasun" in architectures()
    spec = importlib.util.spec_from_file_location("llb200_build", str(__import__("tests.conftest", fromlist=["PKG"]).PKG / "build.py"))
    build = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(build)
    stems = build.FAMILY_SOURCES["Livasun"]
    assert all((build.CSRC / f"{s}.cu").exists() for s in stems)
    assert {"decay_scan", "short_conv", "rotary_attn", "moe_ops"} <= set(stems) and "window_attn" not in stems
