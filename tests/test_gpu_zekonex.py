"""Zekonex on the GPU against the float64 oracle (oracle/zekonex.py): whole prompts and the stream after every layer run,
token-by-token decoding, portions down to two tokens, memory that another request used before, batch rows against each alone, sizes
that are 1 and sizes that are odd, loops of every kind, long decoding, greedy generation through ``generate()`` and the trace session.
Every comparison is against the oracle run on the WHOLE sequence without any memory."""
import numpy as np
import pytest
import torch

from oracle import zekonex as O
from tests.util_zekonex import (TOL32, agrees, attn, case_mixed, case_odd, case_one_kind, case_ones, case_wide, delta, ff, latent, load, model_cfg,
                                random_weights, rel_err, run_schedule, write_model)

pytestmark = pytest.mark.gpu

T_LONG = 45


def fixture_of(case, name, n_tokens, seed):
    @pytest.fixture(scope="module")
    def fx(tmp_path_factory):
        cfg, W = case()
        folder = write_model(tmp_path_factory.mktemp(name), cfg, W)
        toks = np.random.RandomState(seed).randint(0, cfg["vocab"], size=n_tokens).tolist()
        return cfg, W, folder, toks, O.forward(cfg, W, toks)
    return fx


mixed = fixture_of(case_mixed, "mixed", T_LONG, 7)
ones = fixture_of(case_ones, "ones", 23, 8)
odd = fixture_of(case_odd, "odd", 31, 9)
wide = fixture_of(case_wide, "wide", 210, 10)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_whole_prompt_and_every_layer_run(mixed, dtype):
    """A looped layer counts in every pass; the vector that opens a pass is not in the stream the layer before it leaves."""
    cfg, W, folder, toks, want = mixed
    m = load(folder, dtype)
    streams = []
    m.layer_probe = lambda i, x: streams.append(x.double().cpu().numpy().copy())
    got = run_schedule(m, toks, [len(toks)], 64)[0]
    _, want_streams = O.forward(cfg, W, toks, return_layers=True)
    assert len(streams) == len(want_streams) == 12
    for i, (g, w) in enumerate(zip(streams, want_streams)):
        assert agrees(g, w, dtype), f"stream after run {i}: {rel_err(g, w)}"
    assert agrees(got, want, dtype), rel_err(got, want)
    m.layer_probe = None
    assert agrees(run_schedule(m, toks, [len(toks)], 64)[0], want, dtype)       # the sum and the next norm in one launch


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_token_by_token_equals_prefill(mixed, dtype):
    cfg, W, folder, toks, want = mixed
    m = load(folder, dtype)
    got = run_schedule(m, toks, [1] * len(toks), 64)[0]        # the first tokens of a sequence included
    assert agrees(got, want, dtype), rel_err(got, want)
    got = run_schedule(m, toks, [len(toks) - 20] + [1] * 20, 64)[0]
    assert agrees(got, want, dtype), rel_err(got, want)


@pytest.mark.parametrize("portions", [[2] * 22 + [1], [3, 2, 7, 1, 1, 11, 2, 5, 13], [44, 1], [1, 44], [5, 40], [1, 1, 1, 2, 40]])
def test_portions_of_any_size(mixed, portions):
    cfg, W, folder, toks, want = mixed
    m = load(folder, torch.float32)
    assert rel_err(run_schedule(m, toks, portions, 64)[0], want) < TOL32


def test_prompts_the_model_cuts_itself(mixed):
    cfg, W, folder, toks, want = mixed
    for portion in (1, 2, 7, 44):
        m = load(folder, torch.float32, prefill_portion=portion)
        assert rel_err(run_schedule(m, toks, [30] + [1] * 15, 64)[0], want) < TOL32


def test_logits_only_where_asked(mixed):
    cfg, W, folder, toks, want = mixed
    m = load(folder, torch.float32)
    idx = torch.tensor([toks], device="cuda")
    m.reset_cache()
    assert m(idx[:, :20], 64, torch.arange(20), out_rows=[]).shape == (1, 0, cfg["vocab"])
    got = m(idx[:, 20:], 64, torch.arange(20, T_LONG), out_rows=[0, 7, 24]).double().cpu().numpy()[0]
    assert rel_err(got, want[[20, 27, 44]]) < TOL32


def test_a_new_request_reuses_the_memory_of_an_ended_one(mixed):
    """Nothing is cleared between requests: state and rows of the ended request are still there when the next one starts."""
    cfg, W, folder, toks, want = mixed
    m = load(folder, torch.float32)
    other = np.random.RandomState(9).randint(0, cfg["vocab"], size=40).tolist()
    run_schedule(m, other, [33] + [1] * 7, 64)                       # fills the memory and captures the step graph
    ptr = m.states[0].data_ptr()
    for portions in ([T_LONG], [1] * T_LONG, [20] + [1] * 25):
        got = run_schedule(m, toks, portions, 64)[0]
        assert m.states[0].data_ptr() == ptr
        assert rel_err(got, want) < TOL32


def test_memory_full_of_nan_is_never_read(mixed):
    cfg, W, folder, toks, want = mixed
    for dtype in (torch.float32, torch.bfloat16):
        m = load(folder, dtype)
        m._begin(1, 64, True)
        for t in m.states + m.kv_caches:
            t.fill_(float("nan"))
        for portions in ([T_LONG], [1] * 5 + [40]):
            assert agrees(run_schedule(m, toks, portions, 64)[0], want, dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_batch_rows_equal_each_alone(mixed, dtype):
    cfg, W, folder, toks, want = mixed
    m = load(folder, dtype)
    other = np.random.RandomState(10).randint(0, cfg["vocab"], size=T_LONG).tolist()
    want_other = O.forward(cfg, W, other)
    got = run_schedule(m, [toks, other], [17, 2, 1, 1, 24], 64)
    assert agrees(got[0], want, dtype) and agrees(got[1], want_other, dtype), (rel_err(got[0], want), rel_err(got[1], want_other))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_sizes_that_are_one(ones, dtype):
    cfg, W, folder, toks, want = ones
    m = load(folder, dtype)
    for portions in ([len(toks)], [1] * len(toks), [2] * 11 + [1]):
        got = run_schedule(m, toks, portions, 32)[0]
        assert agrees(got, want, dtype), rel_err(got, want)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_sizes_that_are_odd(odd, dtype):
    cfg, W, folder, toks, want = odd
    m = load(folder, dtype)
    for portions in ([len(toks)], [9] + [1] * 22, [2, 3, 5, 7, 11, 3]):
        got = run_schedule(m, toks, portions, 32)[0]
        assert agrees(got, want, dtype), rel_err(got, want)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_wide_heads_and_prompts_of_several_chunks(wide, dtype):
    """bf16 prompts take the tensor-core forms (attention from 16 tokens on, the delta rule from 64); shorter portions and single
    tokens the others: chunk edges inside portions, portions that end inside chunks."""
    cfg, W, folder, toks, want = wide
    m = load(folder, dtype)
    for portions in ([210], [70, 17, 123], [130] + [1] * 80, [16, 3, 64, 65, 2, 60]):
        got = run_schedule(m, toks, portions, 220)[0]
        assert agrees(got, want, dtype), rel_err(got, want)
    other = np.random.RandomState(20).randint(0, cfg["vocab"], size=210).tolist()
    got = run_schedule(m, [toks, other], [150, 60], 220)
    assert agrees(got[0], want, dtype) and agrees(got[1], O.forward(cfg, W, other), dtype)


@pytest.mark.parametrize("kind", ["delta", "attention", "latent_attention"])
def test_models_with_one_kind_of_mixer(kind, tmp_path):
    """Rings without recurrent state, recurrent state without rings."""
    cfg, W = case_one_kind(kind)
    folder = write_model(tmp_path / kind, cfg, W)
    toks = np.random.RandomState(13).randint(0, cfg["vocab"], size=26).tolist()
    want = O.forward(cfg, W, toks)
    m = load(folder, torch.float32)
    for portions in ([26], [1] * 26, [11, 2, 13]):
        assert rel_err(run_schedule(m, toks, portions, 32)[0], want) < TOL32


@pytest.mark.parametrize("loop", [None, (0, 3, 1), (0, 3, 2), (0, 1, 4), (2, 3, 3), (1, 2, 2)])
def test_loops(loop, tmp_path):
    """No loop, one pass over everything, single layers several times; in one step and decoded."""
    cfg = model_cfg(23, 24, [(delta(2, 1, 8, 8), ff(12)), (attn(2, 1, 8, 8, rot=(4, 30.0)), None), (latent(2, 8, 4, 8, 12), ff(8))], loop=loop)
    W = random_weights(cfg, 31)
    folder = write_model(tmp_path / "loop", cfg, W)
    toks = np.random.RandomState(15).randint(0, 23, size=20).tolist()
    want = O.forward(cfg, W, toks)
    m = load(folder, torch.float32)
    for portions in ([20], [1] * 20, [2, 7, 11]):
        assert rel_err(run_schedule(m, toks, portions, 32)[0], want) < TOL32


@pytest.mark.parametrize("kind", ["delta", "attention", "latent_attention"])
def test_a_far_token_reaches_the_end(kind, tmp_path):
    """Two sequences that differ in their second token only: 400 tokens later the logits still differ as the oracle's do - through
    the memory of a slow decay, or through the keys - in one pass, in portions and decoded."""
    mix = {"delta": delta(2, 2, 16, 8), "attention": attn(2, 1, 16, 8, rot=(8, 1e4)), "latent_attention": latent(2, 8, 4, 8, 16)}[kind]
    cfg = model_cfg(31, 24, [(mix, ff(16)), (mix, None)])
    W = random_weights(cfg, 21, qk_gain=2.5)
    if kind == "delta":
        for i in (0, 1):
            W[f"l{i}.mix.A_log"][:], W[f"l{i}.mix.b"][:] = -9.0, 0.25 * W[f"l{i}.mix.b"]
    for i in (0, 1):
        W[f"l{i}.mix.o"] *= 4.0
    folder = write_model(tmp_path / "far", cfg, W)
    toks = np.random.RandomState(14).randint(0, 30, size=401).tolist()
    toks[1], toks[-1] = 30, 30                                    # a token of its own, met again by the last one
    alt = list(toks)
    alt[1] = 3
    want = [O.forward(cfg, W, t)[-1] for t in (toks, alt)]
    gap = np.abs(want[0] - want[1]).max()
    assert gap > 1e-3 * np.abs(want[0]).max()
    m = load(folder, torch.float32)
    for portions in ([401], [100, 3, 2, 296], [380] + [1] * 21):
        got = [run_schedule(m, t, portions, 512)[0][-1] for t in (toks, alt)]
        for g, w in zip(got, want):
            assert rel_err(g, w) < TOL32
        assert np.abs((got[0] - got[1]) - (want[0] - want[1])).max() < 0.05 * gap


def test_long_decoding(mixed):
    cfg, W, folder, _, _ = mixed
    toks = np.random.RandomState(11).randint(0, cfg["vocab"], size=150).tolist()
    want = O.forward(cfg, W, toks)
    m = load(folder, torch.float32)
    got = run_schedule(m, toks, [20] + [1] * 130, 256)[0]
    assert rel_err(got, want) < TOL32


def test_forward_without_kept_memory_leaves_the_memory_alone(mixed):
    cfg, W, folder, toks, want = mixed
    m = load(folder, torch.float32)
    idx = torch.tensor([toks], device="cuda")
    m.reset_cache()
    a = m(idx[:, :30], 64, torch.arange(30))
    probe = m(idx[:, :12]).double().cpu().numpy()[0]             # no positions: scratch memory
    b = m(idx[:, 30:], 64, torch.arange(30, T_LONG))
    assert rel_err(probe, want[:12]) < TOL32
    assert rel_err(torch.cat([a, b], 1).double().cpu().numpy()[0], want) < TOL32


def test_positions_beyond_the_first_rotation_table(mixed):
    """A longer sequence grows the tables of the turns and drops the captured steps that read the old ones."""
    cfg, W, folder, toks, want = mixed
    m = load(folder, torch.float32)
    run_schedule(m, toks, [30] + [1] * 15, 64)
    n = m._rope_len
    got = run_schedule(m, toks, [30] + [1] * 15, n + 7)[0]
    assert m._rope_len >= n + 7 and rel_err(got, want) < TOL32


def test_greedy_generation_through_generate(mixed):
    import generate as G

    cfg, W, folder, toks, _ = mixed
    m = G.load_model(folder, None, torch.device("cuda"), torch.float32)
    prompt = torch.tensor(toks[:9], device="cuda")
    out = G.generate(m, prompt, 12, temperature=1.0, top_k=1).tolist()
    m.reset_cache()
    seq = list(toks[:9])
    for _ in range(12):
        seq.append(int(np.argmax(O.forward(cfg, W, seq)[-1])))
    assert out == seq


def test_trace_session_frees_and_reuses(mixed):
    from lit_llama.trace import TraceSession

    cfg, W, folder, toks, want = mixed
    m = load(folder, torch.float32)
    s = TraceSession(m, 64)
    other = np.random.RandomState(12).randint(0, cfg["vocab"], size=21).tolist()
    assert s.step([{"id": "a", "tokens": other[:20], "want": []}]) is None
    s.step([{"id": "a", "tokens": other[20:], "want": [0]}], end=["a"])
    rows = [s.step([{"id": "b", "tokens": toks[:10], "want": [0, 9]}]),
            s.step([{"id": "b", "tokens": toks[10:12], "want": [1]}]),
            s.step([{"id": "b", "tokens": toks[12:13], "want": [0]}]),
            s.step([{"id": "b", "tokens": toks[13:], "want": [T_LONG - 14]}], end=["b"])]
    got = torch.cat(rows).double().cpu().numpy()
    assert rel_err(got, want[[0, 9, 11, 12, T_LONG - 1]]) < TOL32
