"""The mechanisms Zekonex adds, each alone against its float64 statement (oracle/zekonex.py): RMS norm with the residual sum, a
branch's bias and a vector that joins the stream; softmax attention with interleaved rotation and a constant sink in its fp32 and
tensor-core forms (far keys, first tokens, key ranges split over blocks); the gated delta rule walked token by token and in chunks on
tensor cores (chunk edges, portions, states handed on, keys that repeat, decays of zero and one); latent attention with two-term
weights; clamped units with biases into strided rows.  Inputs are made so that a fault shows: one key takes the whole weight, one
memory is read back hundreds of tokens later, the same key is written again and again."""
import math

import numpy as np
import pytest
import torch

from oracle import zekonex as O
from tests.util_zekonex import bf16

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
    assert np.isfinite(got).all()
    assert np.abs(got - want).max() < tol * max(1.0, np.abs(want).max()), np.abs(got - want).max()


# ------------------------------------------------------------------ stream and feed-forward
@pytest.mark.parametrize("E", [1, 6, 64, 200, 2047, 2048, 3000, 4096, 8192, 9000])
@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_sum_and_rms_norm(E, dtype):
    from lit_llama.stepping import add_rms_norm

    r = np.random.RandomState(E)
    M = 5
    x, a, w, bias, step = r.randn(M, E) + 0.5, r.randn(M, E), r.randn(E), r.randn(E), r.randn(E)
    xs, x0 = dev(x), rounded(x, torch.float32)
    ad, wd, bd, sd = dev(a, dtype), dev(w), dev(bias), dev(step)
    out = torch.empty((M, E), dtype=dtype, device="cuda")
    tol = 1e-5 if dtype == torch.float32 else TOL[dtype]
    add_rms_norm(xs, ad, 0.75, bd, sd, wd, 1e-3, out, dtype)
    nx = x0 + 0.75 * (rounded(a, dtype) + rounded(bias, torch.float32)) + rounded(step, torch.float32)
    close(xs, nx, 1e-6)
    close(out, O.unit_rms(nx, 1e-3) * w, tol)
    kept = xs.clone()
    add_rms_norm(xs, None, 1.0, None, None, wd, 1e-3, out, dtype)        # nothing to add: the stream stays
    assert torch.equal(xs, kept)
    add_rms_norm(xs, ad, 0.5, None, None, None, 1e-3, None, dtype)       # only the sum
    nx = nx + 0.5 * rounded(a, dtype)
    close(xs, nx, 1e-6)
    add_rms_norm(xs, None, 1.0, None, sd, wd, 1e-3, out, dtype)          # only a vector joins
    nx = nx + rounded(step, torch.float32)
    close(xs, nx, 1e-6)
    close(out, O.unit_rms(nx, 1e-3) * w, tol)


@pytest.mark.parametrize("F,lead,pitch", [(8, 16, 32), (24, 8, 40), (7, 3, 20), (1, 0, 8), (130, 6, 140)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_clamped_unit_with_biases_into_strided_rows(F, lead, pitch, dtype):
    """Pre-activations far beyond the clamps on both sides; what lies around the written columns stays."""
    from lit_llama.feed_forward import ClampedUnit

    r = np.random.RandomState(F)
    M, E = 9, 12
    u = ClampedUnit(E, F, 0.8, "cuda")
    W = {n: r.randn(s) for n, s in (("gate.b", F), ("up.b", F), ("down.b", E))}
    u.load(lambda n: dev(W[n]))
    proj = rounded(3 * r.randn(M, lead + 2 * F), dtype)
    rows = torch.full((M, pitch), 9.0, dtype=dtype, device="cuda")
    u(dev(proj, dtype)[:, lead:], rows[:, lead: lead + F])
    want = O.clamped_unit(proj[:, lead:lead + F] + W["gate.b"], proj[:, lead + F:] + W["up.b"], 0.8)
    close(rows[:, lead: lead + F], want, TOL[dtype])
    around = torch.cat([rows[:, :lead], rows[:, lead + F:]], 1)
    assert bool((around == 9.0).all())


# ------------------------------------------------------------------ softmax attention
def mixer(E, H, G, d, e, rot, scale, W, dtype):
    from lit_llama.rotary import RotarySpec
    from lit_llama.softmax_attention import SoftmaxAttention, SoftmaxAttentionSpec

    m = SoftmaxAttention(SoftmaxAttentionSpec(E, H, G, d, e, scale, 1e-5, rotary=RotarySpec.from_dict(rot, d), gate=False,
                                              rot_layout="interleaved", fixed_sink=0.0), dtype, "cuda")
    m.load(lambda s: dev(W[s]))
    return m


def run_attention(m, x, portions, dtype, splits=1, first=0):
    """``x [T, E]`` through the whole mixer in portions, the ring as long as the sequence."""
    T = len(x)
    caches = [torch.full(s, float("nan"), dtype=dtype, device="cuda") for s in m.cache_shapes(1, first + T)]
    xd, out, at = dev(x, dtype), [], 0
    for n in portions:
        out.append(m(xd[at:at + n], 1, n, pos(at, at + n), caches, None, splits))
        at += n
    return torch.cat(out)


@pytest.mark.parametrize("H,G,d,e,dims", [(4, 2, 16, 16, 16), (3, 3, 6, 10, 2), (6, 1, 40, 24, 24), (2, 2, 72, 136, 36), (1, 1, 1, 1, 0), (8, 2, 200, 8, 64)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_attention_mixer(H, G, d, e, dims, dtype):
    r = np.random.RandomState(H * 100 + d)
    E, T = 24, 75
    W = {n: rounded(r.randn(k, E) / np.sqrt(E), dtype) for n, k in (("q", H * d), ("k", G * d), ("v", G * e))}
    W["o"] = rounded(r.randn(E, H * e) / np.sqrt(H * e), dtype)
    rot = {"dims": dims, "base": 100.0} if dims else None
    m_cfg = {"heads": H, "kv_heads": G, "rot": rot, "scale": 1.3 / math.sqrt(d)}
    x = rounded(2 * r.randn(T, E), dtype)
    want = O.attention(x, W, "", m_cfg, np.arange(T))
    m = mixer(E, H, G, d, e, rot, m_cfg["scale"], W, dtype)
    for portions, splits in (([T], 1), ([1] * T, 3), ([40, 2, 17, 16], 1), ([T - 1, 1], 7)):
        close(run_attention(m, x, portions, dtype, splits), want, 5e-5 if dtype == torch.float32 else 5e-2)


@pytest.mark.parametrize("dtype,portions,splits", [
    (torch.float32, [600], 1), (torch.float32, [599, 1], 1), (torch.float32, [599, 1], 16), (torch.bfloat16, [600], 1),
    (torch.bfloat16, [500, 100], 1), (torch.bfloat16, [599, 1], 5)])
def test_a_far_key_found_through_its_turn(dtype, portions, splits):
    """All keys are the same up to their position's turn, and one query is the one that the turn of a key 596 tokens back undoes;
    pairs (i, i + dims/2) instead of neighbours, or a position that is off by one, would point it at another key."""
    H, G, d, e, T, far = 2, 1, 64, 32, 600, 3
    base = 40.0
    k = np.repeat(np.random.RandomState(1).randn(1, d), T, axis=0) * 2.0
    # query i is the key turned back by its own distance to `far`: after both turns they agree
    q = np.zeros((T, H, d))
    q[:] = k[0]
    q[T - 1] = O.turn(k[None, :1], [far - (T - 1)], d, base)[0, 0]
    v = np.random.RandomState(2).randn(T, e)
    E = H * d + d + e
    x = np.concatenate([q.reshape(T, -1), k, v], axis=1)
    W = {"q": np.eye(E)[:H * d], "k": np.eye(E)[H * d:H * d + d], "v": np.eye(E)[H * d + d:], "o": np.eye(H * e)}
    x = rounded(x, dtype)
    rot = {"dims": d, "base": base}
    m = mixer(E, H, G, d, e, rot, 0.35, dict(W, o=np.concatenate([W["o"], np.zeros((E - H * e, H * e))])), dtype)
    got = host(run_attention(m, x, portions, dtype, splits))[-1, :H * e].reshape(H, e)
    want = O.causal_softmax(O.turn(x[:, :H * d].reshape(T, H, d), np.arange(T), d, base), O.turn(x[:, None, H * d:H * d + d], np.arange(T), d, base),
                            x[:, None, H * d + d:], 0.35, 1.0)[-1]
    close(got, want, 1e-4 if dtype == torch.float32 else 3e-2)
    assert np.abs(want - x[far, H * d + d:]).max() < 0.2, "the far key should carry most of the weight"


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_sink_at_the_first_tokens(dtype):
    """Keys whose scores are around and far below zero: the first token's output is v / (1 + e^-s), not v; and far above zero the sink
    vanishes."""
    r = np.random.RandomState(3)
    H, d, e, T, E = 2, 8, 8, 40, 24
    W = {n: rounded(r.randn(16, E) / 5, dtype) for n in "qkv"}
    W["o"] = np.eye(E)[:, :16]
    x = rounded(r.randn(T, E), dtype)
    for scale in (0.01, -30.0, 30.0):
        m = mixer(E, H, 2, d, e, None, scale, W, dtype)
        q, k, v = (rounded(x @ W[n].T, dtype).reshape(T, 2, 8) for n in "qkv")
        want = O.causal_softmax(q, k, v, scale, 1.0).reshape(T, -1)
        for portions in ([T], [1] * T, [2, 20, 18]):
            close(host(run_attention(m, x, portions, dtype))[:, :16], want, 2e-4 if dtype == torch.float32 else 3e-2)
        s = scale * (q[0] * k[0]).sum(-1)
        assert np.allclose(want[0].reshape(2, 8), v[0] / (1 + np.exp(-s))[:, None])


# ------------------------------------------------------------------ gated delta rule
def delta_case(r, T, H, G, n, p, dtype, repeat=False):
    q, k, v = (rounded(r.randn(T, c), dtype) for c in (G * n, G * n, H * p))
    if repeat:                        # three directions only: what is written for a key meets what was written for it before
        k = rounded(r.randn(3, G * n), dtype)[r.randint(3, size=T)]
    a, b = rounded(2 * r.randn(T, H), dtype), rounded(2 * r.randn(T, H) + 1, dtype)
    return q, k, v, a, b, rounded(r.uniform(-4, 0, H), torch.float32), rounded(r.uniform(-3, 1, H), torch.float32)


def delta_want(q, k, v, a, b, dt_bias, a_log, H, G, n, p, qs, eps=1e-6):
    T = len(q)
    unit = lambda t: t / np.sqrt((t * t).sum(-1, keepdims=True) + eps)
    g, beta = O.delta_gates(a, b, dt_bias, a_log)
    o, S = O.delta_memory(unit(q.reshape(T, G, n)) * qs, unit(k.reshape(T, G, n)), v.reshape(T, H, p), g, beta)
    return o.reshape(T, -1), S


def run_delta(case, H, G, n, p, portions, dtype, qs, state, eps=1e-6):
    from lit_llama.recurrence import delta_scan

    q, k, v, a, b, dt_bias, a_log = case
    at, got = 0, []
    gates = dev(np.concatenate([a, b], axis=1), dtype)
    qkv = dev(np.concatenate([q, k, v], axis=1), dtype)
    dtb, al = dev(dt_bias), dev(a_log)
    for m in portions:
        x = qkv[at:at + m]
        got.append(delta_scan(x, 0, x, G * n, x, 2 * G * n, gates[at:at + m], 0, H, dtb, al, eps, qs, state, pos(at, at + m), 1, m, H, G, n, p))
        at += m
    return torch.cat(got)


@pytest.mark.parametrize("H,G,n,p", [(4, 2, 8, 8), (3, 3, 10, 5), (6, 2, 40, 24), (2, 1, 72, 136), (1, 1, 1, 1), (2, 2, 130, 3), (2, 1, 300, 3),
                                     (40, 20, 64, 64)])
@pytest.mark.parametrize("repeat", [False, True])
@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_rule_walk_in_portions(H, G, n, p, repeat, dtype):
    r = np.random.RandomState(n + p)
    T, qs = 41, 0.3
    case = delta_case(r, T, H, G, n, p, dtype, repeat)
    want, S = delta_want(*case, H, G, n, p, qs)
    state = torch.full((1, H, n, p), float("nan"), device="cuda")
    for portions in ([T], [1] * T, [17, 2, 1, 21]):
        close(run_delta(case, H, G, n, p, portions, dtype, qs, state), want, 2e-5)
        close(state[0], S, 2e-5)


@pytest.mark.parametrize("H,G,n,p", [(2, 1, 8, 8), (4, 2, 16, 24), (3, 3, 40, 64), (4, 2, 64, 72), (2, 2, 128, 136), (6, 1, 104, 16), (16, 8, 64, 136), (40, 20, 24, 96)])
@pytest.mark.parametrize("repeat", [False, True])
def test_delta_rule_in_chunks(H, G, n, p, repeat):
    """Chunk edges, last chunks that are not full, steps that begin inside a sequence, a decay of zero and one of one in the middle of a
    chunk, write strengths near one and near zero, keys that repeat within a chunk (the triangular system is far from diagonal)."""
    from lit_llama import _native as N

    r = np.random.RandomState(n + p)
    T, qs, bf = 300, 0.3, torch.bfloat16
    case = delta_case(r, T, H, G, n, p, bf, repeat)
    case[3][100], case[3][170], case[3][200:230] = 90.0, -90.0, -90.0       # forget everything; nothing; nothing for a while
    case[4][210:240] = 30.0                                                 # full strength: what was stored is replaced
    case[4][240:250] = -30.0
    want, S = delta_want(*case, H, G, n, p, qs)
    stride = 2 * G * n + H * p
    for portions in ([300], [64, 236], [70, 5, 65, 1, 159], [127, 128, 45]):
        for m in portions:
            assert bool(N.call_ret("ll_delta_chunked_supported", N.LL_BF16, m, n, p, stride, stride, stride)) == (m >= 64)
        state = torch.full((1, H, n, p), float("nan"), device="cuda")
        close(run_delta(case, H, G, n, p, portions, bf, qs, state), want, 5e-5)      # (16 bits where fp32 factors meet each other)
        close(state[0], S, 5e-5)
    assert N.call_ret("ll_delta_chunk_error") == 0              # no wait for a copy ran out


def test_chunks_and_walk_agree_on_identical_keys(monkeypatch):
    """Every token writes under the same key with nearly full strength and hardly any decay: the inverse of the triangular system
    has entries that a power series would only reach through huge cancelling terms."""
    import lit_llama.recurrence as R

    H, G, n, p, T, bf = 2, 1, 32, 16, 256, torch.bfloat16
    r = np.random.RandomState(0)
    case = list(delta_case(r, T, H, G, n, p, bf))
    case[1] = np.repeat(case[1][:1], T, axis=0)
    case[3][:], case[4][:] = -20.0, 4.0
    want, S = delta_want(*case, H, G, n, p, 1.0)
    for chunks in (True, False):
        monkeypatch.setattr(R, "USE_CHUNKS", chunks)
        state = torch.full((1, H, n, p), float("nan"), device="cuda")
        close(run_delta(case, H, G, n, p, [T], bf, 1.0, state), want, 5e-5)
        close(state[0], S, 5e-5)


@pytest.mark.parametrize("dtype,portions", [(torch.float32, [700]), (torch.bfloat16, [700]), (torch.bfloat16, [333, 2, 365]), (torch.bfloat16, [65, 635])])
def test_a_memory_read_back_hundreds_of_tokens_later(dtype, portions):
    """One key is written once at token 65 and read at the end; the tokens between write under keys orthogonal to it."""
    H, G, n, p, T = 1, 1, 16, 8, 700
    q, k, v = np.zeros((T, n)), np.zeros((T, n)), np.zeros((T, p))
    k[:, 1 + np.arange(T) % 15] = 0.0
    k[np.arange(T), 1 + np.arange(T) % 15] = 2.0
    v[:] = 1.0
    k[65], v[65] = np.eye(n)[0] * 3.0, np.arange(1, p + 1)
    for t in (64, 65, 66, T - 1):
        q[t] = np.eye(n)[0] * 5.0
    a, b = np.full((T, 1), -60.0), np.full((T, 1), 30.0)                     # no decay, full strength
    state = torch.full((1, H, n, p), float("nan"), device="cuda")
    y = host(run_delta((q, k, v, a, b, np.zeros(1), np.zeros(1)), H, G, n, p, portions, dtype, 1.0, state, eps=0.0))
    for t in (65, 66, T - 1):
        close(y[t], np.arange(1, p + 1), 1e-5)
    assert np.abs(y[64]).max() < 1e-6


def test_delta_batch_rows_and_zero_vectors():
    """Rows of a batch differ; a query or key of zeros has no direction (the constant inside the root keeps it at zero)."""
    from lit_llama.recurrence import delta_scan

    H, G, n, p, T, B, bf = 4, 2, 24, 40, 130, 3, torch.bfloat16
    r = np.random.RandomState(5)
    cases = [delta_case(r, T, H, G, n, p, bf) for _ in range(B)]
    for c in cases:
        c[0][[5, 70]], c[1][[6, 66, 129]] = 0.0, 0.0
    dt_bias, a_log = cases[0][5], cases[0][6]
    want = [delta_want(*c[:5], dt_bias, a_log, H, G, n, p, 0.5) for c in cases]
    qkv = dev(np.concatenate([np.concatenate(c[:3], axis=1) for c in cases]), bf)
    gates = dev(np.concatenate([np.concatenate(c[3:5], axis=1) for c in cases]), bf)
    dtb, al = dev(dt_bias), dev(a_log)
    for dtype in (bf, torch.float32):
        state = torch.full((B, H, n, p), float("nan"), device="cuda")
        x, gg = qkv.to(dtype), gates.to(dtype)
        y = host(delta_scan(x, 0, x, G * n, x, 2 * G * n, gg, 0, H, dtb, al, 1e-6, 0.5, state, pos(0, T), B, T, H, G, n, p)).reshape(B, T, -1)
        for i in range(B):
            close(y[i], want[i][0], 5e-5)
            close(state[i], want[i][1], 5e-5)


@pytest.mark.parametrize("H,G,n,p,taps", [(4, 2, 16, 24, 4), (3, 1, 7, 5, 1), (2, 2, 40, 8, 6), (4, 2, 16, 24, 2)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_mixer(H, G, n, p, taps, dtype):
    from lit_llama.recurrence import GatedDeltaMixer, GatedDeltaSpec

    r = np.random.RandomState(n + taps)
    E, T, eps = 24, 147, 1e-4
    W = {s: rounded(r.randn(c, E) / 4, dtype) for s, c in (("q", G * n), ("k", G * n), ("v", H * p), ("g", H * p), ("a", H), ("b", H))}
    for s, c in (("q", G * n), ("k", G * n), ("v", H * p)):
        W[s + ".conv"] = bf16(0.6 * r.randn(c, taps))
    W["A_log"], W["dt_bias"], W["norm"] = bf16(r.uniform(-3, 1, H)), bf16(r.uniform(-3, 0, H)), bf16(1 + 0.3 * r.randn(p))
    W["o"] = rounded(r.randn(E, H * p) / np.sqrt(H * p), dtype)
    mix = GatedDeltaMixer(GatedDeltaSpec(E, H, G, n, p, taps, eps), dtype, "cuda")
    mix.load(lambda s: dev(W[s]))
    x = rounded(r.randn(T, E), dtype)
    want = O.delta(x, W, "", {"heads": H, "kv_heads": G, "dim": n, "vdim": p}, eps)
    for portions in ([T], [1] * 20 + [127], [9, 1, 2, 70, 65]):
        state = [torch.full(s, float("nan"), device="cuda") for s in mix.state_shapes(1)]
        got, at = [], 0
        for m in portions:
            got.append(mix(dev(x[at:at + m], dtype), 1, m, pos(at, at + m), state))
            at += m
        close(torch.cat(got), want, 1e-4 if dtype == torch.float32 else 6e-2)


# ------------------------------------------------------------------ latent attention
@pytest.mark.parametrize("H,n,rd,e,R", [(4, 16, 8, 16, 32), (3, 5, 6, 7, 9), (8, 24, 16, 40, 136), (2, 8, 2, 8, 8), (33, 8, 8, 8, 16), (2, 16, 32, 8, 264)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_mixer_without_gate(H, n, rd, e, R, dtype):
    from lit_llama.latent_attention import LatentAttention, LatentAttentionSpec
    from lit_llama.rotary import RotarySpec

    r = np.random.RandomState(R + H)
    E, T, eps = 24, 90, 1e-4
    W = {"q": r.randn(H * (n + rd), E) / 4, "dkv": r.randn(R + rd, E) / 4, "dkv.norm": bf16(1 + 0.3 * r.randn(R)), "uk": r.randn(H * n, R) / np.sqrt(R),
         "uv": r.randn(H * e, R) / np.sqrt(R), "o": r.randn(E, H * e) / np.sqrt(H * e)}
    W = {k: w if k == "dkv.norm" else rounded(w, dtype) for k, w in W.items()}
    rot, sc = {"dims": rd, "base": 90.0}, 3.0 / (n + rd)
    x = rounded(2 * r.randn(T, E), dtype)
    want = O.latent_attention(x, W, "", {"heads": H, "dim": n, "rot_dim": rd, "kv_rank": R, "scale": sc, "rot": rot}, eps, np.arange(T))
    mix = LatentAttention(LatentAttentionSpec(E, H, n, rd, e, R, None, sc, eps=eps, gate="none", rotary=RotarySpec.from_dict(rot), exact_weights=True),
                          dtype, "cuda")
    mix.load(lambda s: dev(W[s]).cpu())
    rope = mix.spec.rope_table(T, "cuda")
    for portions, splits in (([T], 1), ([1] * T, 3), ([40, 2, 31, 17], 1), ([T - 1, 1], 16)):
        cache = torch.full((1, T, R + rd), float("nan"), dtype=dtype, device="cuda")
        got, at = [], 0
        for m in portions:
            got.append(mix(dev(x[at:at + m], dtype), 1, m, pos(at, at + m), rope, cache, splits))
            at += m
        close(torch.cat(got), want, 5e-5 if dtype == torch.float32 else 5e-2)


@pytest.mark.parametrize("R,rd,H,T", [(64, 16, 4, 200), (256, 64, 16, 130), (512, 64, 16, 70), (24, 8, 1, 90)])
@pytest.mark.parametrize("window,splits", [(0, 1), (33, 1), (0, 4)])
def test_weights_as_two_terms(R, rd, H, T, window, splits):
    """The same step with one and with two terms, on values of one sign and nearly equal weights, so that the rounding of the weights
    does not average out against anything else: two terms leave only the rounding of the result."""
    import lit_llama._native as N

    r = np.random.RandomState(R)
    bf = torch.bfloat16
    q_lat, c = rounded(r.randn(H, T, R) * 0.3 / np.sqrt(R), bf), rounded(1 + 0.1 * r.randn(T, R), bf)
    ql, proj, cache = dev(q_lat, bf), torch.zeros((T, H * rd), dtype=bf, device="cuda"), dev(np.concatenate([c, np.zeros((T, rd))], 1)[None], bf)
    rope = torch.zeros((T, rd // 2, 2), device="cuda")
    want = np.zeros((H, T, R))
    for i in range(T):
        lo = max(0, i - window + 1) if window else 0
        s = q_lat[:, i] @ c[lo:i + 1].T
        w = np.exp(s - s.max(-1, keepdims=True))
        want[:, i] = (w / w.sum(-1, keepdims=True)) @ c[lo:i + 1]
    err = {}
    for terms in (1, 2):
        out = torch.empty_like(ql)
        scratch = torch.empty(max(4, N.call_ret("ll_latent_attn_scratch_bytes", T, H, R, splits) // 4), device="cuda")
        N.call("ll_latent_attn_terms", N.ptr(ql), T * R, R, N.ptr(proj), H * rd, 0, rd, -1, N.ptr(rope), N.ptr(pos(0, T)), N.ptr(cache), N.ptr(out),
               T * R, R, N.LL_BF16, 1, T, H, R, rd, rd, T, window, 1.0, splits, terms, N.ptr(scratch), N.stream())
        torch.cuda.synchronize()
        err[terms] = np.abs(host(out) - want).max()
    assert err[2] < 2.0 ** -8 * 1.01 * np.abs(want).max() and err[2] <= err[1] + 1e-9, err
