"""The mechanisms Livasun adds, each alone against its float64 statement (oracle/livasun.py): layer norm with the residual sum,
norms per head with query temperature, value mixing and ring append, softmax attention with a bias linear in the distance
in its fp32 and tensor-core forms (window edges, far keys, first tokens, rings that wrap, key ranges split over blocks), the
recurrence with constant decays, long parts in the gated norm, the corrected sigmoid router, squared-relu experts in their
three forms, silu-gated layers.  Inputs are made so that a fault shows: one key takes the whole weight just inside or just
outside a window, one memory is read back hundreds of tokens later."""
import math

import numpy as np
import pytest
import torch

from oracle import livasun as O
from tests.util_livasun import bf16

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
TOL = {torch.float32: 2e-5, torch.bfloat16: 1.5e-2}


def dev(a, dtype=torch.float32):
    return None if a is None else torch.tensor(np.asarray(a, dtype=np.float64), dtype=dtype, device="cuda")


def host(t):
    return t.double().cpu().numpy()


def pos(a, b):
    return torch.arange(a, b, dtype=torch.int32, device="cuda")


def rounded(a, dtype):
    return host(dev(a, dtype))


def close(got, want, tol):
    got = host(got) if torch.is_tensor(got) else got
    assert np.abs(got - want).max() < tol * max(1.0, np.abs(want).max()), np.abs(got - want).max()


# ------------------------------------------------------------------ stream
@pytest.mark.parametrize("E", [1, 6, 64, 200, 2047, 2048, 3000, 4096, 8192, 9000])
@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_sum_and_layer_norm(E, dtype):
    """Rows held in registers (multiples of 4 up to 8192) and in shared memory; a mean far from zero, so that a variance taken
    from the mean of the squares would be off."""
    from lit_llama.stepping import add_layer_norm

    r = np.random.RandomState(E)
    M = 5
    x, a, w, b = r.randn(M, E) + 40.0, r.randn(M, E), r.randn(E), r.randn(E)
    xs, x0 = dev(x), rounded(x, torch.float32)
    ad, wd, bd = dev(a, dtype), dev(w), dev(b)
    out = torch.empty((M, E), dtype=dtype, device="cuda")
    add_layer_norm(xs, ad, 0.75, wd, bd, 1e-3, out, dtype)
    nx = x0 + 0.75 * rounded(a, dtype)
    close(xs, nx, 1e-6)
    close(out, O.layer_norm(nx, w, b, 1e-3), 1e-4 if dtype == torch.float32 else TOL[dtype])
    kept = xs.clone()
    add_layer_norm(xs, None, 1.0, wd, bd, 1e-3, out, dtype)              # nothing to add: the stream stays
    assert torch.equal(xs, kept)
    add_layer_norm(xs, ad, 1.0, None, None, 1e-3, None, dtype)           # only the sum
    close(xs, nx + rounded(a, dtype), 1e-6)


# ------------------------------------------------------------------ attention
def append(q, k, v, first, lam, wq, wk, eps, temp, p0, ring, G, dtype, rot=None):
    """ll_qk_head_append on one step of q [T, H, d], k [T, G, d], v [T, G, e]; returns (q out, key ring, value ring)."""
    import lit_llama._native as N
    from lit_llama.rotary import RotarySpec

    T, H, d = q.shape
    e = v.shape[2]
    row = np.concatenate([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], axis=1)
    proj, fd = dev(row, dtype), dev(first.reshape(T, -1), dtype) if first is not None else None
    wqd, wkd, pd = dev(wq), dev(wk), pos(p0, p0 + T)
    freq = RotarySpec.from_dict(rot).frequencies("cuda")
    qo = torch.empty((T, H * d), dtype=dtype, device="cuda")
    kc = torch.full((1, ring, G * d), 9.0, dtype=dtype, device="cuda")
    vc = torch.full((1, ring, G * e), 9.0, dtype=dtype, device="cuda")
    n = row.shape[1]
    N.call("ll_qk_head_append", N.ptr(proj), n, N.ptr_at(proj, H * d), n, N.ptr_at(proj, (H + G) * d), n, N.ptr(fd), G * e, float(lam),
           N.dtype_code(dtype), N.ptr(wqd), N.ptr(wkd), float(eps), N.ptr(freq), rot["dims"] if rot else 0, float(temp[0]), temp[1],
           N.ptr(pd), N.ptr(qo), N.ptr(kc), N.ptr(vc), 1, T, H, G, d, e, ring, N.stream())
    torch.cuda.synchronize()
    return host(qo).reshape(T, H, d), host(kc)[0].reshape(ring, G, d), host(vc)[0].reshape(ring, G, e)


@pytest.mark.parametrize("H,G,d,e", [(3, 1, 10, 6), (4, 4, 48, 32), (1, 1, 1, 1), (9, 3, 64, 5), (2, 1, 129, 16), (16, 2, 256, 64)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_head_norm_temperature_value_mix_and_append(H, G, d, e, dtype):
    """Positions around a step of the temperature, far from zero; rows land in their ring slots; heads of very different size,
    so that a norm over the wrong numbers shows."""
    r = np.random.RandomState(d)
    T, ring, every, eps = 9, 11, 7, 1e-3
    p0 = 5 * 7 * 31 - 3                                                   # floor((p + 1) / every) steps inside the portion
    gain = np.exp(2 * r.randn(H))[:, None]
    q, k, v = r.randn(T, H, d) * gain, r.randn(T, G, d) * 3, r.randn(T, G, e)
    first, lam = r.randn(T, G, e), 0.3125
    wq, wk = 1 + 0.3 * r.randn(d), 1 + 0.3 * r.randn(d)
    qo, kc, vc = append(q, k, v, first, lam, wq, wk, eps, (0.6, every), p0, ring, G, dtype)
    q, k, v, first = (rounded(t, dtype) for t in (q, k, v, first))
    p = np.arange(p0, p0 + T)
    want_q = O.unit_rms(q, eps) * wq * O.temperature(p, 0.6, every)[:, None, None]
    close(qo, want_q, TOL[dtype])
    close(kc[p % ring], O.unit_rms(k, eps) * wk, TOL[dtype])
    close(vc[p % ring], O.mix_values(v, first, lam), TOL[dtype])
    untouched = [s for s in range(ring) if s not in set(p % ring)]
    assert (kc[untouched] == 9.0).all() and (vc[untouched] == 9.0).all()
    qo, kc, vc = append(q, k, v, None, lam, wq, wk, eps, (0.6, 0), p0, ring, G, dtype)        # neither temperature nor mix
    close(qo, O.unit_rms(q, eps) * wq, TOL[dtype])
    assert np.array_equal(vc[p % ring], v)


def test_head_norm_with_rotation_and_without_norm():
    from oracle.tebodra import rotate

    r = np.random.RandomState(3)
    T, H, G, d, e = 7, 5, 2, 20, 4
    rot = {"base": 100.0, "dims": 12}
    q, k, v = r.randn(T, H, d), r.randn(T, G, d), r.randn(T, G, e)
    w = 1 + 0.3 * r.randn(d)
    p = np.arange(300, 300 + T)
    qo, kc, _ = append(q, k, v, None, 0.0, w, w, 1e-4, (0.0, 0), 300, 8, G, torch.float32, rot)
    close(qo, rotate(O.unit_rms(q, 1e-4) * w, rot, p), 5e-5)
    close(kc[p % 8], rotate(O.unit_rms(k, 1e-4) * w, rot, p), 5e-5)
    qo, _, _ = append(q, k, v, None, 0.0, None, None, 1e-4, (0.5, 4), 300, 8, G, torch.float32, rot)
    close(qo, rotate(q * O.temperature(p, 0.5, 4)[:, None, None], rot, p), 5e-5)


def run_attention(q, k, v, first, ring, scale, dtype, slopes=None, cap=0.0, window=0, splits=1, form=0):
    """The queries at ``first``..L-1 run in ONE step against a ring of ``ring`` slots (position j in slot j % ring)."""
    import lit_llama._native as N

    L, H, d = q.shape
    G, e = k.shape[1], v.shape[2]
    T = L - first
    kh, vh = np.full((1, ring, G * d), np.nan), np.full((1, ring, G * e), np.nan)
    for j in range(L):
        kh[0, j % ring], vh[0, j % ring] = k[j].reshape(-1), v[j].reshape(-1)
    kc, vc, qd, sd, pd = dev(kh, dtype), dev(vh, dtype), dev(q[first:].reshape(T, H * d), dtype), dev(slopes), pos(first, L)
    y = torch.empty((T, H * e), dtype=dtype, device="cuda")
    scratch = torch.empty(max(4, N.call_ret("ll_softmax_attn_scratch_bytes", T, H, e, splits) // 4), dtype=torch.float32, device="cuda")
    N.call("ll_softmax_attn_biased", N.ptr(qd), H * d, None, 0, N.ptr(kc), N.ptr(vc), N.dtype_code(dtype), N.ptr(pd), None, N.ptr(sd),
           float(scale), float(cap), 1, T, H, G, d, e, window, 0, ring, splits, form, 1, 0.0, 1.0, 0.0, N.ptr(scratch), N.ptr(y), N.stream())
    torch.cuda.synchronize()
    return host(y).reshape(T, H, e)


def rand_qkv(r, L, H, G, d, e, gain=1.0):
    return bf16(r.randn(L, H, d) * gain), bf16(r.randn(L, G, d) * gain), bf16(r.randn(L, G, e))


@pytest.mark.parametrize("H,G,d,e", [(4, 2, 16, 16), (3, 3, 6, 10), (6, 1, 40, 24), (2, 2, 72, 136), (1, 1, 1, 1), (8, 2, 200, 8)])
@pytest.mark.parametrize("window", [0, 1, 9, 33])
def test_biased_attention_fp32(H, G, d, e, window):
    r = np.random.RandomState(H * 100 + d + window)
    L = 50
    q, k, v = rand_qkv(r, L, H, G, d, e)
    scale = 1.7 / math.sqrt(d)
    want = O.biased_attention(q, k, v, scale, O.slopes(H), window or None)
    for first, splits in ((0, 1), (30, 1), (49, 1), (49, 3), (47, 16)):
        ring = L if not window else window - 1 + (L - first)             # as short as the look-back allows: it wraps
        got = run_attention(q, k, v, first, ring, scale, torch.float32, O.slopes(H), 0.0, window, splits)
        close(got, want[first:], 2e-5)


@pytest.mark.parametrize("d,e", [(16, 16), (32, 8), (48, 64), (72, 40), (96, 96), (128, 128)])
@pytest.mark.parametrize("window", [0, 40, 64, 3])
def test_biased_attention_tensor_core_form(d, e, window):
    """bf16 steps of 16 tokens or more: tiles of 64 queries, window edges inside tiles, a last tile that is not full, heads
    narrower than the padded tile, a ring that wraps; beside the fp32 form on the same bf16 inputs."""
    r = np.random.RandomState(d + e + window)
    L, H, G = 171, 4, 2
    q, k, v = rand_qkv(r, L, H, G, d, e)
    scale = 1.7 / math.sqrt(d)
    want = O.biased_attention(q, k, v, scale, O.slopes(H), window or None)
    for first in (0, 41, 155):
        ring = L if not window else window - 1 + (L - first)
        for form in (0, 1):
            got = run_attention(q, k, v, first, ring, scale, torch.bfloat16, O.slopes(H), 0.0, window, form=form)
            close(got, want[first:], TOL[torch.bfloat16])


def test_the_bias_enters_before_the_cap():
    r = np.random.RandomState(4)
    L, H, d = 40, 2, 16
    q, k, v = rand_qkv(r, L, H, 1, d, 8)
    slope = np.array([0.5, 0.125])
    want = np.zeros((L, H, 8))
    for i in range(L):
        for h in range(H):
            s = 3.0 * np.tanh((k[:i + 1, 0] @ q[i, h] - slope[h] * (i - np.arange(i + 1))) / 3.0)
            w = np.exp(s - s.max())
            want[i, h] = (w / w.sum()) @ v[:i + 1, 0]
    for dtype in DTYPES:
        close(run_attention(q, k, v, 0, L, 1.0, dtype, slope, 3.0), want, TOL[dtype])


def spike(L, H, G, d, e, at, query, r, size=7.0):
    """Small random keys, except that key ``at`` and query ``query`` point the same way with a large product."""
    q, k, v = rand_qkv(r, L, H, G, d, e, gain=0.05)
    u = np.zeros(d)
    u[0] = size
    k[at, :] = u
    q[query, :] = u
    return q, k, v


@pytest.mark.parametrize("dtype,first,splits", [(torch.float32, 0, 1), (torch.float32, 60, 1), (torch.float32, 69, 1), (torch.float32, 69, 3),
                                                (torch.float32, 69, 16), (torch.bfloat16, 0, 1), (torch.bfloat16, 50, 1), (torch.bfloat16, 69, 4)])
def test_a_key_just_inside_and_just_outside_the_window(dtype, first, splits):
    """Query 69 with a window of 16 sees 54..69.  A key at 54 that matches it takes nearly all the weight; the same key at 53 is
    not seen at all.  In a prompt's portion and decoded alone, whatever the split of the keys."""
    r = np.random.RandomState(5)
    L, H, G, d, e, window = 70, 4, 2, 16, 16, 16
    for at, seen in ((54, True), (53, False)):
        q, k, v = spike(L, H, G, d, e, at, 69, r)
        got = run_attention(q, k, v, first, L, 1.0, dtype, O.slopes(H), 0.0, window, splits)[-1]
        close(got, O.biased_attention(q, k, v, 1.0, O.slopes(H), window)[-1], TOL[dtype])
        near = np.abs(got - v[at][np.arange(H) // (H // G)]).max()
        assert (near < 0.05) == seen, (at, near)


@pytest.mark.parametrize("dtype,first,splits", [(torch.float32, 0, 1), (torch.float32, 699, 1), (torch.float32, 699, 16), (torch.bfloat16, 600, 1)])
def test_a_far_key_among_hundreds(dtype, first, splits):
    """A distance of 696 and slopes of 1/16 and 1/256: the far key still wins, but by what the bias leaves of its score."""
    r = np.random.RandomState(6)
    L, H, G, d, e = 700, 2, 1, 32, 32
    q, k, v = spike(L, H, G, d, e, 3, 699, r)
    got = run_attention(q, k, v, first, L, 1.0, dtype, O.slopes(H), splits=splits)[-1]
    want = O.biased_attention(q, k, v, 1.0, O.slopes(H))[-1]
    close(got, want, TOL[dtype])
    assert np.abs(want[1] - v[3, 0]).max() < 0.05


# ------------------------------------------------------------------ recurrence with constant decays
@pytest.mark.parametrize("H,n,p", [(3, 10, 8), (4, 48, 32), (2, 16, 5), (1, 1, 1), (2, 130, 3), (2, 300, 3), (2, 128, 64), (40, 64, 64)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_constant_decay_recurrence_in_portions(H, n, p, dtype):
    from lit_llama.recurrence import decay_scan_constant

    r = np.random.RandomState(n + p)
    T = 41
    decay = np.concatenate([[0.0, 1.0], r.uniform(0.5, 1.0, H)])[-H:] if H > 2 else r.uniform(0.5, 1.0, H)
    proj = rounded(r.randn(T, H * (2 * n + p) + 3), dtype)
    act = rounded(O.silu(proj), dtype) if dtype == torch.bfloat16 else O.silu(proj)
    for silu in (True, False):
        a = act if silu else proj
        q, k, v = a[:, :H * n].reshape(T, H, n), a[:, H * n:2 * H * n].reshape(T, H, n), a[:, 2 * H * n:2 * H * n + H * p].reshape(T, H, p)
        want = O.constant_decay_memory(q, k, v, decay).reshape(T, -1)
        state = torch.full((1, H, n, p), float("nan"), device="cuda")
        dd, pd = dev(decay), dev(proj, dtype)
        for portions in ([T], [1] * T, [17, 2, 1, 21]):
            got, at = [], 0
            for m in portions:
                got.append(decay_scan_constant(pd[at:at + m], 0, H * n, 2 * H * n, dd, silu, 1.0, state, pos(at, at + m), 1, m, H, H, n, p))
                at += m
            close(torch.cat(got), want, 2e-5 if dtype == torch.float32 or not silu else 2e-3)    # (a bf16 tie of the activation may round either way)


def test_a_memory_read_back_hundreds_of_tokens_later():
    """What token 0 wrote, decayed 700 times, read by one query; across portions, in a batch whose rows differ."""
    from lit_llama.recurrence import decay_scan_constant

    T, n, p = 700, 8, 4
    proj = np.zeros((2, T, 2 * n + p))
    proj[0, 0, n + 3], proj[0, 0, 2 * n:], proj[0, -1, 3] = 1.0, [1.0, 2.0, 3.0, 4.0], 1.0
    proj[1, 5, n + 3], proj[1, 5, 2 * n:], proj[1, -1, 3] = 1.0, [-1.0, 0.5, 3.0, 4.0], 2.0
    decay = dev([0.999])
    state = torch.full((2, 1, n, p), float("nan"), device="cuda")
    got = []
    for lo, hi in ((0, 333), (333, 335), (335, T)):
        part = dev(proj[:, lo:hi].reshape(2 * (hi - lo), -1))
        got.append(decay_scan_constant(part, 0, n, 2 * n, decay, False, 1.0, state, pos(lo, hi), 2, hi - lo, 1, 1, n, p).reshape(2, hi - lo, p))
    y = host(torch.cat(got, 1))
    assert np.abs(y[:, :-1]).max() == 0.0
    close(y[0, -1], 0.999 ** 699 * np.array([1.0, 2.0, 3.0, 4.0]), 1e-4)
    close(y[1, -1], 2 * 0.999 ** 694 * np.array([-1.0, 0.5, 3.0, 4.0]), 1e-4)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,d,e", [(2, 8, 12), (4, 32, 96), (1, 5, 7)])
def test_lightning_mixer(H, d, e, dtype):
    from lit_llama.recurrence import ConstantDecayAttention, ConstantDecaySpec

    r = np.random.RandomState(H + e)
    E, T, eps = 24, 19, 1e-4
    decay = r.uniform(0.5, 0.999, H)
    W = {n: rounded(r.randn(H * (e if n in "vg" else d), E) / 4, dtype) for n in "qkvg"}
    W["o"], W["norm"] = rounded(r.randn(E, H * e) / 5, dtype), bf16(1 + 0.3 * r.randn(H * e))
    mix = ConstantDecayAttention(ConstantDecaySpec(E, H, d, e, decay, eps), dtype, "cuda")
    mix.load(lambda s: dev(W[s]))
    x = rounded(r.randn(T, E), dtype)
    want = O.lightning(x, W, "", {"heads": H, "decay": decay}, eps)
    state = [torch.full(s, float("nan"), device="cuda") for s in mix.state_shapes(1)]
    got = torch.cat([mix(dev(x[:12], dtype), 1, 12, pos(0, 12), state), mix(dev(x[12:13], dtype), 1, 1, pos(12, 13), state),
                     mix(dev(x[13:], dtype), 1, T - 13, pos(13, T), state)])
    close(got, want, 5e-5 if dtype == torch.float32 else 4e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,P,Nst,G,norm_groups", [(4, 8, 16, 2, 2), (8, 80, 16, 1, 2), (2, 6, 10, 2, 1), (6, 128, 8, 3, 1)])
def test_state_space_mixer_with_long_and_short_norm_parts(H, P, Nst, G, norm_groups, dtype):
    from lit_llama.recurrence import StateSpaceMixer, StateSpaceSpec

    r = np.random.RandomState(P)
    E, T, eps, inner = 24, 17, 1e-4, H * P
    C = inner + 2 * G * Nst
    W = {"in": rounded(r.randn(inner + C + H, E) / 4, dtype), "conv": bf16(0.6 * r.randn(C, 3)), "conv.b": bf16(0.2 * r.randn(C)),
         "dt_bias": bf16(r.uniform(-2, 1, H)), "A_log": bf16(r.uniform(-2, 1, H)), "D": bf16(r.randn(H)),
         "norm": bf16(1 + 0.3 * r.randn(inner)), "o": rounded(r.randn(E, inner) / np.sqrt(inner), dtype)}
    mix = StateSpaceMixer(StateSpaceSpec(E, H, P, Nst, G, norm_groups, 3, eps), dtype, "cuda")
    mix.load(lambda s: dev(W[s]))
    x = rounded(r.randn(T, E), dtype)
    want = O.mamba2(x, W, "", {"heads": H, "vdim": P, "state": Nst, "groups": G, "norm_groups": norm_groups}, eps)
    state = [torch.full(s, float("nan"), device="cuda") for s in mix.state_shapes(1)]
    got = torch.cat([mix(dev(x[:9], dtype), 1, 9, pos(0, 9), state), mix(dev(x[9:10], dtype), 1, 1, pos(9, 10), state),
                     mix(dev(x[10:], dtype), 1, T - 10, pos(10, T), state)])
    close(got, want, 5e-5 if dtype == torch.float32 else 4e-2)


# ------------------------------------------------------------------ router, experts, dense layers
@pytest.mark.parametrize("X,top,count,keep", [(16, 4, 4, 3), (6, 2, 3, 2), (9, 2, 3, 1), (4, 2, 4, 2), (8, 3, 1, 1), (1, 1, 1, 1), (40, 5, 8, 2)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_corrected_sigmoid_router(X, top, count, keep, dtype):
    """Corrections of both signs, choice scores below zero (a group that is out counts as minus infinity, not as 0)."""
    from lit_llama.moe import MoE, MoESpec

    r = np.random.RandomState(X)
    M, E = 65, 24
    moe = MoE(MoESpec(E, X, top, 8, float("inf"), router_bias=False, score="sigmoid", groups=count, keep_groups=keep, group_top=2,
                      correction=True, weight_scale=2.25, unit="relu2"), dtype, "cuda")
    w, corr = rounded(r.randn(X, E), torch.float32), rounded(r.uniform(-2.0, 0.3, X), torch.float32)
    moe.w_router.copy_(dev(w))
    moe.correction.copy_(dev(corr))
    x = rounded(r.randn(M, E), dtype)
    idx, wts, offsets, perm = moe.route(dev(x, dtype))
    widx, wwts = O.route(x, w, corr, top, 2.25, count, keep)
    gi = idx.cpu().numpy()
    assert np.array_equal(np.sort(gi, 1), np.sort(widx, 1))
    close(np.take_along_axis(host(wts), np.argsort(gi, 1), 1), np.take_along_axis(wwts, np.argsort(widx, 1), 1), 1e-5)
    off, pm, flat = offsets.cpu().numpy(), perm.cpu().numpy(), gi.reshape(-1)
    assert off[-1] == M * top and sorted(pm.tolist()) == list(range(M * top))
    for e in range(X):
        assert (flat[pm[off[e]:off[e + 1]]] == e).all()


@pytest.mark.parametrize("M,E,ff,shared", [(1, 32, 16, 8), (5, 30, 11, 7), (70, 32, 16, None), (700, 64, 72, 40)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_squared_relu_experts(M, E, ff, shared, dtype, monkeypatch):
    """Single tokens, odd sizes, many rows; in bfloat16 with aligned rows also the tcgen05 kernels, whatever the step's size."""
    import lit_llama.moe as MOE
    from lit_llama import _native as N

    r = np.random.RandomState(M)
    X, top = 6, 2
    cfgf = {"router": {"experts": X, "top": top, "scale": 1.5, "groups": {"count": 3, "keep": 2}}, "shared": {"ff": shared} if shared else None}
    moe = MOE.MoE(MOE.MoESpec(E, X, top, ff, float("inf"), shared_ff=shared, shared_gate=False, router_bias=False, score="sigmoid", groups=3,
                              keep_groups=2, group_top=2, correction=True, weight_scale=1.5, unit="relu2"), dtype, "cuda")
    W = {"router": rounded(r.randn(X, E), torch.float32), "correction": rounded(r.uniform(-1, 0.2, X), torch.float32)}
    for q, n in [(f"e{e}.", ff) for e in range(X)] + ([("shared.", shared)] if shared else []):
        W[q + "up"], W[q + "down"] = rounded(r.randn(n, E) * 1.5 / np.sqrt(E), dtype), rounded(r.randn(E, n) / np.sqrt(n), dtype)
    moe.load(lambda s: dev(W[s]))
    x = rounded(r.randn(M, E), dtype)
    want = O.moe_ff(x, W, "", cfgf)
    close(moe(dev(x, dtype)), want, TOL[dtype] * 3)
    if dtype == torch.bfloat16 and E % 8 == 0 and ff % 8 == 0:
        monkeypatch.setattr(MOE, "TC_MIN_ROWS", 1)
        monkeypatch.setattr(MOE, "TC_MIN_ROWS_PER_EXPERT", 0)
        assert moe.takes_tensor_cores(M * top, dev(x, dtype))
        close(moe(dev(x, dtype)), want, TOL[dtype] * 3)
        assert N.call_ret("ll_moe_tc_error") == 0


@pytest.mark.parametrize("M,E,ff", [(1, 24, 40), (9, 30, 13), (130, 64, 96)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_silu_gated_dense_layer(M, E, ff, dtype):
    from lit_llama.feed_forward import DenseFF

    r = np.random.RandomState(ff)
    W = {"gate": rounded(r.randn(ff, E) * 2 / np.sqrt(E), dtype), "up": rounded(r.randn(ff, E) / np.sqrt(E), dtype),
         "down": rounded(r.randn(E, ff) / np.sqrt(ff), dtype)}
    f = DenseFF(E, ff, "silu_glu", dtype, "cuda")
    f.load(lambda s: dev(W[s]))
    x = rounded(r.randn(M, E), dtype)
    close(f(dev(x, dtype)), O.dense_ff(x, W, ""), TOL[dtype] * 2)


# ------------------------------------------------------------------ the recurrences in chunks on tensor cores
def chunk_case(r, T, H, G, n, p, low=0.5):
    q, k, v = (bf16(r.randn(T, c)) for c in (G * n, G * n, H * p))
    a = r.uniform(low, 1.0, (T, H))
    return q, k, v, a, r.uniform(0.1, 1.5, (T, H)), r.randn(H)


def chunk_want(q, k, v, a, ks, skip, qs, H, G, n, p):
    T = len(q)
    y = np.zeros((T, H, p))
    for h in range(H):
        g, S = h // (H // G), np.zeros((n, p))
        for t in range(T):
            S = a[t, h] * S + ks[t, h] * np.outer(k[t, g * n:(g + 1) * n], v[t, h * p:(h + 1) * p])
            y[t, h] = qs * (S.T @ q[t, g * n:(g + 1) * n]) + skip[h] * v[t, h * p:(h + 1) * p]
    return y.reshape(T, H * p), S


@pytest.mark.parametrize("H,G,n,p", [(2, 1, 8, 8), (4, 2, 16, 24), (3, 3, 40, 64), (2, 1, 64, 72), (2, 2, 128, 136), (6, 1, 104, 16)])
@pytest.mark.parametrize("low", [0.0, 0.9])
def test_chunked_recurrence_against_the_walk(H, G, n, p, low):
    """Chunk edges, last chunks that are not full, a step that begins inside a sequence, decays near zero and near one, a decay of
    exactly zero in the middle of a chunk; outputs and the state handed on agree with float64 to fp32 accuracy."""
    import lit_llama.recurrence as R

    r = np.random.RandomState(n + p)
    T = 300
    q, k, v, a, ks, skip = chunk_case(r, T, H, G, n, p, low)
    a[100] = 0.0
    a[170, 0] = 1e-30
    want, S = chunk_want(q, k, v, a, ks, skip, 0.5, H, G, n, p)
    bfl = torch.bfloat16
    for portions in ([300], [64, 236], [70, 5, 65, 1, 159], [127, 128, 45]):
        state = torch.full((1, H, n, p), float("nan"), device="cuda")
        got, at = [], 0
        for m in portions:
            ops = [dev(q[at:at + m], bfl), dev(k[at:at + m], bfl), dev(v[at:at + m], bfl)]
            assert R.takes_chunks(m, H, n, p, *[(o, 0) for o in ops]) == (m >= 64)
            got.append(R.decay_scan(ops[0], 0, ops[1], 0, ops[2], 0, dev(a[at:at + m]), False, dev(ks[at:at + m]), dev(skip), 0.5, state,
                                    pos(at, at + m), 1, m, H, G, n, p))
            at += m
        close(torch.cat(got), want, 3e-5)                       # (the read-out's weights carry 16 bits)
        close(state[0, H - 1], S, 2e-6)


@pytest.mark.parametrize("H,n,p", [(3, 32, 48), (2, 128, 128), (4, 8, 8)])
def test_chunked_constant_decay_with_silu(H, n, p, monkeypatch):
    """The same step walked and in chunks: the same activations bit for bit, so that outputs differ by summation only; a batch."""
    import lit_llama.recurrence as R

    r = np.random.RandomState(p)
    B, T = 2, 200
    proj = dev(r.randn(B * T, H * (2 * n + p)), torch.bfloat16)
    decay = dev([0.0, 0.999, 0.7, 1.0][:H])
    outs = []
    for chunks in (True, False):
        monkeypatch.setattr(R, "USE_CHUNKS", chunks)
        state = torch.full((B, H, n, p), float("nan"), device="cuda")
        y = R.decay_scan_constant(proj, 0, H * n, 2 * H * n, decay, True, 1.0, state, pos(0, T), B, T, H, H, n, p)
        outs.append((host(y), host(state)))
    close(outs[0][0], outs[1][0], 3e-5)
    close(outs[0][1], outs[1][1], 2e-6)
    act = rounded(O.silu(host(proj)[:T]), torch.bfloat16)
    want = O.constant_decay_memory(act[:, :H * n].reshape(T, H, n), act[:, H * n:2 * H * n].reshape(T, H, n),
                                   act[:, 2 * H * n:].reshape(T, H, p), host(decay)).reshape(T, -1)
    close(outs[0][0][:T], want, 2e-3)                           # (a bf16 tie of the activation may round either way)


def test_a_memory_read_back_across_many_chunks():
    """Decay one: what a token wrote is read back 700 tokens and ten chunks later to fp32 accuracy, and nothing before it."""
    import lit_llama.recurrence as R

    T, n, p = 777, 16, 8
    q, k, v = np.zeros((T, n)), np.zeros((T, n)), np.zeros((T, p))
    k[65, 3], v[65] = 1.0, np.arange(1, p + 1)
    q[64, 3], q[65, 3], q[66, 3], q[-1, 3] = 1.0, 1.0, 1.0, 1.0
    state = torch.full((1, 1, n, p), float("nan"), device="cuda")
    bfl = torch.bfloat16
    y = host(R.decay_scan(dev(q, bfl), 0, dev(k, bfl), 0, dev(v, bfl), 0, dev(np.ones((T, 1))), False, None, None, 1.0, state, pos(0, T), 1, T,
                          1, 1, n, p))
    for t in (65, 66, T - 1):
        close(y[t], np.arange(1, p + 1), 1e-6)
    assert np.abs(y[:65]).max() == 0.0 and np.abs(y[67:-1]).max() == 0.0
