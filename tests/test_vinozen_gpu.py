"""Vinozen on the GPU against the plain implementation (tests/plain/vinozen_plain.py): every mechanism alone,
then the engine under every way of cutting requests into steps, in 32-bit and in bfloat16."""
import os

import numpy as np
import pytest

import schedules
from plain import vinozen_plain as plain
from test_engine_gpu import run_steps
from vinozen_cases import CASES, attention, case, dense, layer, make_folder, mamba2, random_tokens
from vinozen_cases import moe as moe_spec

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ["float32", "bfloat16"]
FP32_TOL = 3e-4
PAGE = 64


def torch_dtype(name):
    import torch
    return {"float32": torch.float32, "bfloat16": torch.bfloat16}[name]


def dev(a, dtype):
    import torch
    return torch.tensor(np.asarray(a), dtype=dtype, device="cuda")


def f64(t):
    return t.double().cpu().numpy()


def close(dtype, loose=2e-2):
    return dict(rtol=3e-5, atol=3e-5) if dtype == "float32" else dict(rtol=loose, atol=loose)


def packed(lengths):
    """seq_start and token_seq of a step whose sequences bring `lengths` tokens (all positive)."""
    start = np.concatenate([[0], np.cumsum(lengths)]).astype(np.int32)
    seq = np.concatenate([np.full(n, i) for i, n in enumerate(lengths)]).astype(np.int32)
    return start, seq


class Bound:
    """A part with its tensors, for running it alone on `N` tokens."""

    def __init__(self, family, kind, params, weights, T, N, **ctx):
        import torch
        from qwen3_b200.config import PartSpec
        from qwen3_b200.engine.context import Scratch
        from qwen3_b200.parts import build_part
        from qwen3_b200.weights.upload import TensorDict
        self.part = build_part(family, PartSpec(kind, params))
        tensors = weights(self.part.weight_specs("l0."))
        self.weights = {n[len("l0."):]: f64(t) for n, t in tensors.items()}
        self.part.bind(TensorDict(dict(tensors), self.part.weight_specs("l0."), T, torch.device("cuda"), lambda n: None), "l0.", T,
                       torch.device("cuda"))
        self.ctx = type("Ctx", (), dict(n_tokens=N, scratch=Scratch("cuda", guard=True), dtype=T, device=torch.device("cuda"), **ctx))


# ============================================================================ mechanisms, one at a time
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [5, 50, 64, 132, 516, 2048, 2052, 4096, 6000, 9000])
def test_layer_norm_of_a_branch_and_the_residual_sum(dtype, size):
    """A branch far from zero mean: a norm without centring, or with a variance that cancels, is far off."""
    import torch
    from qwen3_b200.csrc import ops
    from qwen3_b200.parts.norm import LayerNorm, RMSNorm
    rng = np.random.default_rng(size)
    T, N = torch_dtype(dtype), 7
    stream = dev(rng.standard_normal((N, size)) * 3 + 2, torch.float32)
    branch = dev(rng.standard_normal((N, size)) + 30 * rng.standard_normal((N, 1)), T)

    def norm(cls):
        part = cls(size, 1e-5)
        part.weight = dev(1 + 0.3 * rng.standard_normal(size), torch.float32)
        return part
    a, b, r = norm(LayerNorm), norm(LayerNorm), norm(RMSNorm)
    idx = dev([3, 0, 6, 3], torch.int32)
    for post in (None, a, r):
        for pre in (None, "round", b, r):
            if post is None and pre is None:
                continue
            x, out = stream.clone(), torch.full((N, size), 9.0, dtype=T, device="cuda")
            picked = torch.full((4, size), 9.0, dtype=T, device="cuda")
            ops.settle_norm(x, branch if post else None, post, pre, out if pre else None)
            add = 0.0 if post is None else (plain.layer_norm(f64(branch), f64(a.weight), 1e-5) if post is a
                                            else plain.rms_unit(f64(branch), 1e-5) * f64(r.weight))
            want = f64(stream) + add
            assert np.allclose(f64(x), want, rtol=1e-4, atol=2e-4)
            if pre:
                normed = want if pre == "round" else (plain.layer_norm(want, f64(b.weight), 1e-5) if pre is b
                                                      else plain.rms_unit(want, 1e-5) * f64(r.weight))
                tol = dict(rtol=2e-4, atol=4e-4) if dtype == "float32" else dict(rtol=1e-2, atol=1e-2)
                assert np.allclose(f64(out), normed, **tol)
                y = stream.clone()                               # picked rows: nothing is written to the stream
                ops.settle_norm(y, branch if post else None, post, pre, picked, rows=idx, n_rows=4, compute_dtype=T)
                assert np.allclose(f64(picked), normed[[3, 0, 6, 3]], **tol) and torch.equal(y, stream)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden", [6, 7, 64, 1001, 2048])
def test_embedding_with_sinusoids(dtype, hidden):
    """Positions from the first to far ones: the angle is right to 32-bit rounding everywhere; an id outside the table adds
    nothing."""
    import torch
    from qwen3_b200.parts.embedding import TokenEmbedding
    rng = np.random.default_rng(hidden)
    T, vocab = torch_dtype(dtype), 40
    part = TokenEmbedding(vocab, hidden, scale=2.5, tensor="", positions="sinusoid")
    table = dev(rng.standard_normal((vocab, hidden)), T)
    part.bind({"embed": table}, "embed", T, torch.device("cuda"))
    positions = np.array([0, 1, 2, 63, 64, 4095, 40000, 131071, 1000003])
    ids = np.concatenate([rng.integers(0, vocab, len(positions) - 1), [vocab + 3]])
    out = torch.empty((len(ids), hidden), dtype=torch.float32, device="cuda")
    part.forward(dev(ids, torch.int32), out, dev(positions, torch.int32))
    want = plain.sinusoid(positions, hidden)
    want[:-1] += 2.5 * f64(table)[ids[:-1]]
    assert np.allclose(f64(out), want, rtol=1e-6, atol=2e-6)


def scattered_pages(rng, lengths, heads, width, T, columns=9):
    """A page table in no particular order, and zeroed pages for it."""
    import torch
    n = sum(-(-l // PAGE) for l in lengths)
    order, at = rng.permutation(n), 0
    table = np.full((len(lengths), columns), -1, dtype=np.int32)
    for s, l in enumerate(lengths):
        for pg in range(-(-l // PAGE)):
            table[s, pg] = order[at]
            at += 1
    return table, torch.zeros((n + 1, heads, PAGE, width), dtype=T, device="cuda")


def read_pages(pages, table, s, n):
    """[n, heads, width] of sequence s."""
    p = f64(pages)
    return np.stack([p[table[s, j // PAGE], :, j % PAGE] for j in range(n)])


def fill_pages(pages, table, s, values, T):
    values = dev(values, T)
    for pg in range(-(-len(values) // PAGE)):
        part = values[pg * PAGE:(pg + 1) * PAGE]
        pages[table[s, pg], :, :len(part)] = part.transpose(0, 1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("lengths", [[3, 1, 9], [90, 1, 70]])          # few tokens: a warp a head; many: 16-byte packets where sizes allow
@pytest.mark.parametrize("H,G,d,vd,temp,own", [(4, 2, 16, 24, (0.5, 7), True), (4, 2, 64, 64, (1.0, 64), True), (3, 3, 5, 10, (0.9, 1), True),
                                               (2, 1, 32, 32, None, True), (4, 2, 64, 32, (0.7, 10), False), (3, 1, 11, 11, (0.3, 5), False)])
def test_queries_and_keys_at_unit_rms_with_a_temperature(dtype, lengths, H, G, d, vd, temp, own):
    """One rounding of the normed, warmed query; keys without the temperature; a projection of the queries alone writes no
    page."""
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(d * 10 + H + len(lengths))
    T, eps, pos0 = torch_dtype(dtype), 1e-5, [0, 100, 6]
    start, seq = packed(lengths)
    pos = np.concatenate([np.arange(p, p + n) for p, n in zip(pos0, lengths)]).astype(np.int32)
    N = len(pos)
    rows = dev(rng.standard_normal((N, H * d + (G * (d + vd) if own else 0))) * 5, T)
    table, k_pages = scattered_pages(rng, [p + n for p, n in zip(pos0, lengths)], G, d, T)
    v_pages = torch.zeros(k_pages.shape[:-1] + (vd,), dtype=T, device="cuda")
    ones = torch.ones(d, dtype=torch.float32, device="cuda")
    q = torch.empty((N, H * d), dtype=T, device="cuda")
    ops.qkv_prepare(rows, q, k_pages, v_pages, ones, ones, None, None, dev(seq, torch.int32), dev(pos, torch.int32), dev(table, torch.int32),
                    N, H, G, d, eps, write_kv=own, value_dim=vd, norm_once=True, temperature=temp)
    x = f64(rows)
    qs = plain.rms_unit(x[:, :H * d].reshape(N, H, d), eps)
    if temp:
        qs = qs * plain.query_temperature(pos, *temp)[:, None, None]
    tol = dict(rtol=1e-5, atol=3e-5) if dtype == "float32" else dict(rtol=2 ** -8, atol=1e-5)
    assert np.allclose(f64(q).reshape(N, H, d), qs, **tol)
    if not own:
        assert float(k_pages.abs().max()) == 0.0 and float(v_pages.abs().max()) == 0.0
        return
    ks, vs = plain.rms_unit(x[:, H * d:(H + G) * d].reshape(N, G, d), eps), x[:, (H + G) * d:].reshape(N, G, vd)
    for s, (p, n) in enumerate(zip(pos0, lengths)):
        assert np.allclose(read_pages(k_pages, table, s, p + n)[p:], ks[start[s]:start[s + 1]], **tol)
        assert np.allclose(read_pages(v_pages, table, s, p + n)[p:], vs[start[s]:start[s + 1]], **tol)


def spread(rel, reach):
    """The biases by distance as the kernels take them, [heads, distances], from the plain function."""
    last = next(n for n in range(10 ** 6) if plain.bucket(n, len(rel), reach) == len(rel) - 1)
    return np.stack([rel[plain.bucket(n, len(rel), reach)] for n in range(last + 1)], axis=1)


BIASES = ["lively", "row 0", "row 1", "middle", "before last", "last", "far key"]


def bias_case(rng, H, rows, kind):
    """A table of biases in which one row towers (its stretch's edges show in every query), or a lively one."""
    if kind in ("lively", "far key"):
        return 1.5 * rng.standard_normal((rows, H))
    at = {"row 0": 0, "row 1": 1, "middle": rows // 2, "before last": rows - 2, "last": rows - 1}[kind]
    rel = -2.0 * np.ones((rows, H)) + 0.3 * rng.standard_normal((rows, H))
    rel[at] += 7.0
    return rel


def attention_step(rng, T, H, G, d, vd, lengths, kind):
    """Cached keys and values and queries of every position; with `far key`, one key far back that the last queries ask for."""
    q, k, v = ([rng.standard_normal((n, h, w)) for n in lengths] for h, w in ((H, d), (G, d), (G, vd)))
    if kind == "far key":
        for s, n in enumerate(lengths):
            if n > 20:
                k[s][n // 5] = 3.0 * np.abs(k[s][n // 5])
                q[s][-8:] = np.abs(q[s][-8:])
    table, k_pages = scattered_pages(rng, lengths, G, d, T)
    import torch
    v_pages = torch.zeros(k_pages.shape[:-1] + (vd,), dtype=T, device="cuda")
    for s in range(len(lengths)):
        fill_pages(k_pages, table, s, k[s], T)
        fill_pages(v_pages, table, s, v[s], T)
    return [[f64(dev(x, T)) for x in xs] for xs in (q, k, v)], dev(table, torch.int32), k_pages, v_pages


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,vd,rows,reach", [(4, 2, 16, 32, 8, 40), (3, 3, 5, 10, 7, 12), (2, 1, 32, 16, 32, 200), (1, 1, 8, 8, 2, 3)])
@pytest.mark.parametrize("kind", BIASES)
def test_attention_with_biases_by_distance(dtype, H, G, d, vd, rows, reach, kind):
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(H * 100 + d)
    T, lengths, scale = torch_dtype(dtype), [150, 1, 66], 0.6
    rel, sink = bias_case(rng, H, rows, kind), np.array([1.0, -20.0, 6.0, 2.0])[:H]
    (q, k, v), table, k_pages, v_pages = attention_step(rng, T, H, G, d, vd, lengths, kind)
    start, seq = packed(lengths)
    out = torch.empty((sum(lengths), H * vd), dtype=T, device="cuda")
    ops.attention_generic(dev(np.concatenate(q).reshape(-1, H * d), T), k_pages, v_pages, out, dev(seq, torch.int32),
                          dev(np.concatenate([np.arange(n) for n in lengths]), torch.int32), table, sum(lengths), H, G, d, scale, value_dim=vd,
                          sink=True, sink_values=dev(sink, torch.float32), bias=dev(spread(rel, reach), torch.float32))
    want = np.concatenate([plain.biased_attention(q[s], k[s], v[s], scale, rel, reach, sink) for s in range(3)])
    assert np.allclose(f64(out).reshape(want.shape), want, **close(dtype))


@pytest.mark.parametrize("H,G,d,vd,rows,reach", [(4, 2, 64, 64, 32, 128), (2, 1, 128, 128, 24, 90), (6, 3, 16, 32, 9, 30), (4, 1, 64, 16, 32, 500),
                                                 (16, 1, 32, 32, 2, 3), (2, 2, 128, 64, 16, 64)])
@pytest.mark.parametrize("kind", BIASES)
def test_tiled_attention_with_biases_by_distance(H, G, d, vd, rows, reach, kind):
    """Whole prompts through the tiled kernel and, where the sizes allow it, the tcgen05 kernel; a second portion; single
    tokens through the split decode kernel with 1, 2 and 5 splits."""
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(H * 100 + d)
    T, lengths, scale, atol = torch.bfloat16, [420, 1, 131], 0.3, 3e-2
    rel, sink = bias_case(rng, H, rows, kind), (3.0 * rng.standard_normal(H))
    (q, k, v), table, k_pages, v_pages = attention_step(rng, T, H, G, d, vd, lengths, kind)
    want = [plain.biased_attention(q[s], k[s], v[s], scale, rel, reach, sink) for s in range(3)]
    sinks, bias = dev(sink, torch.float32), dev(spread(rel, reach), torch.float32)
    for first in ([0, 0, 0], [200, 0, 67]):                       # whole prompts; what follows a first portion
        part = [n - f for n, f in zip(lengths, first)]
        start, _ = packed(part)
        rows_q = dev(np.concatenate([q[s][f:] for s, f in enumerate(first)]).reshape(-1, H * d), T)
        meta = (dev(start, torch.int32), dev(first, torch.int32), table, 3, max(part))
        exact = np.concatenate([w[f:] for w, f in zip(want, first)])
        out = torch.full((rows_q.shape[0], H * vd), 9.0, dtype=T, device="cuda")
        ops.attention_capped_prefill(rows_q, k_pages, v_pages, out, *meta, H, G, d, vd, scale, sink=True, sink_values=sinks, bias=bias)
        assert np.allclose(f64(out).reshape(exact.shape), exact, atol=atol)
        if ops.attention_capped_prefill_tc_fits(d, vd, None):
            out.fill_(9.0)
            ops.attention_capped_prefill_tc(rows_q, k_pages, v_pages, out, *meta, rows_q.shape[0], H, G, d, scale, sink=True, sink_values=sinks,
                                            bias=bias)
            assert np.allclose(f64(out).reshape(exact.shape), exact, atol=atol)
            assert ops.tcgen05_status(torch.device("cuda")) == 0
    for at in ([419, 0, 130], [64, 0, 63], [128, 0, 64]):
        rows_q = dev(np.stack([q[s][p] for s, p in enumerate(at)]).reshape(3, H * d), T)
        for splits in (1, 2, 5):
            scratch, out = torch.empty(3 * H * splits * (vd + 2), dtype=torch.float32, device="cuda"), torch.empty((3, H * vd), dtype=T, device="cuda")
            ops.attention_capped_decode(rows_q, k_pages, v_pages, out, scratch, dev([0, 1, 2], torch.int32), dev(at, torch.int32), table, 3, H, G, d, vd,
                                        scale, 0.0, None, True, splits, sink_values=sinks, bias=bias)
            assert np.allclose(f64(out).reshape(3, H, vd), np.stack([want[s][p] for s, p in enumerate(at)]), atol=atol)


def test_biases_that_do_not_fit_are_refused():
    import torch
    from qwen3_b200.csrc import ops
    z = torch.zeros((1, 32), dtype=torch.bfloat16, device="cuda")
    pages = torch.zeros((2, 1, PAGE, 16), dtype=torch.bfloat16, device="cuda")
    i = torch.zeros((1, 4), dtype=torch.int32, device="cuda")
    with pytest.raises(ops.KernelError, match="biases by distance"):
        ops.attention_generic(z, pages, pages, z.clone(), i[0], i[0], i, 1, 2, 1, 16, 1.0, bias=torch.zeros((3, 5), device="cuda"))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,taps,lead", [(24, 4, 0), (24, 2, 8), (64, 3, 64), (13, 4, 0), (40, 5, 16), (16, 1, 0)])
def test_convolution_with_a_bias_and_silu(dtype, C, taps, lead):
    """Columns in the middle of wider rows, portions shorter than the taps, through five steps."""
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(C * 10 + taps)
    T, slots = torch_dtype(dtype), [3, 0, 2]
    w, b = rng.standard_normal((C, taps)), rng.standard_normal(C)
    state = torch.zeros((5, max((taps - 1) * C, 1)), dtype=torch.float32, device="cuda")[:, :(taps - 1) * C]
    seen = [np.zeros((0, C)) for _ in slots]
    for lengths in ([5, 1, 40], [1, 1, 1], [2, 3, 1], [1, 1, 1], [130, 1, 17]):
        start, seq = packed(lengths)
        u = dev(rng.standard_normal((int(start[-1]), lead + C + 8)), T)
        out = torch.empty((u.shape[0], C), dtype=T, device="cuda")
        ops.short_conv(u[:, lead:], dev(w.T.copy(), torch.float32), state, dev(seq, torch.int32), dev(start, torch.int32), dev(slots, torch.int32),
                       out, 3, bias=dev(b, torch.float32), silu=True, single=max(lengths) == 1)
        got = f64(out)
        for s, n in enumerate(lengths):
            seen[s] = np.concatenate([seen[s], f64(u)[start[s]:start[s + 1], lead:lead + C]])
            want = plain.silu(plain.short_convolution(seen[s], f64(dev(w, torch.float32)), f64(dev(b, torch.float32))))
            assert np.allclose(got[start[s]:start[s + 1]], want[-n:], **close(dtype, 1e-2))


SPACES = [(6, 3, 20, 12), (4, 2, 128, 64), (2, 1, 32, 48), (3, 3, 5, 7), (1, 1, 16, 16), (4, 1, 64, 128), (2, 2, 256, 80), (8, 8, 48, 32)]


def space_rows(rng, T, N, H, G, n, vd):
    """Rows of x | B | C as a convolution leaves them, with the columns of each."""
    u = dev(rng.standard_normal((N, H * vd + 2 * G * n)) * np.where(np.arange(H * vd + 2 * G * n) < H * vd, 1.0, n ** -0.25), T)
    at = np.cumsum([H * vd, G * n])
    return u, u[:, :at[0]], u[:, at[0]:at[1]], u[:, at[1]:]


@pytest.mark.parametrize("dtype,H,G,n,vd,chunks", [(dtype, *s, False) for s in SPACES for dtype in DTYPES]
                         + [("bfloat16", *s, True) for s in SPACES if s[2] % 16 == 0 and s[3] % 16 == 0])
def test_state_space_over_unequal_sequences_and_from_its_state(dtype, H, G, n, vd, chunks):
    """Prompts of all lengths around a chunk's edge, portions and single tokens on slots in no particular order; the state in
    columns of a wider row; heads that forget at once and heads that hardly do."""
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(H * 1000 + n + vd)
    T, cells, slots = torch_dtype(dtype), H * n * vd, [4, 0, 5, 2]
    lead = 4 if chunks or n % 2 == 0 else 3                     # whether the rows split into 16-byte packets
    whole = torch.zeros((8, lead + cells + 4 - cells % 4), dtype=torch.float32, device="cuda")
    whole[:, :lead], whole[:, lead + cells:] = 7.0, -7.0
    state = whole[:, lead:lead + cells]
    a_log, dt_bias = np.linspace(-4.0, 3.5, H), rng.standard_normal(H) - 1.0
    skip = rng.standard_normal(H)
    vectors = {k: dev(v, torch.float32) for k, v in (("a_log", a_log), ("dt_bias", dt_bias), ("skip", skip))}
    S = {s: np.zeros((H, n, vd)) for s in slots}
    for lengths in ([1, 63, 130, 64], [65, 1, 2, 40], [1, 1, 1, 1], [200, 1, 33, 3]):
        start, _ = packed(lengths)
        N = int(start[-1])
        u, x, B, C = space_rows(rng, T, N, H, G, n, vd)
        z = dev(rng.standard_normal((N, H)) * 2, torch.float32)
        out = torch.full((N, H * vd), 9.0, dtype=torch.float32, device="cuda")
        args = (C, B, x, state, dev(start, torch.int32), dev(slots, torch.int32), out, 4, H, n, vd)
        if chunks and max(lengths) > 1:
            ops.ssd_prompt(*args, share=H // G, dt_logits=z, max_new=max(lengths), **vectors)
        else:                                                    # single tokens: also the form for them, where rows allow it
            ops.decay_scan(*args, share=H // G, dt_logits=z, **vectors, single=max(lengths) == 1 and ops.state_step_fits(state, vd))
        got, dt = f64(out).reshape(N, H, vd), plain.softplus(f64(z) + f64(vectors["dt_bias"]))
        xs, Bs, Cs = f64(x).reshape(N, H, vd), f64(B).reshape(N, G, n), f64(C).reshape(N, G, n)
        rate = np.exp(f64(vectors["a_log"]))
        for i, slot in enumerate(slots):
            for t in range(start[i], start[i + 1]):
                for h in range(H):
                    g = h // (H // G)
                    S[slot][h] = np.exp(-rate[h] * dt[t, h]) * S[slot][h] + dt[t, h] * np.outer(Bs[t, g], xs[t, h])
                    want = S[slot][h].T @ Cs[t, g] + skip[h] * xs[t, h]
                    assert np.allclose(got[t, h], want, rtol=5e-4, atol=5e-4), (lengths, slot, t - start[i], h)
    final = f64(whole)
    for slot in slots:
        assert np.allclose(final[slot, lead:lead + cells].reshape(H, n, vd), S[slot], rtol=5e-4, atol=5e-4)
    assert np.all(final[:, :lead] == 7.0) and np.all(final[:, lead + cells:] == -7.0) and np.all(final[[1, 3, 6, 7], lead:lead + cells] == 0.0)


@pytest.mark.parametrize("H,G,n,vd", [(4, 2, 128, 64), (2, 1, 32, 48), (3, 3, 16, 128)])
@pytest.mark.parametrize("segments", [None, 2, 3, 7])
def test_long_prompts_of_a_state_space_in_segments(H, G, n, vd, segments):
    """The same numbers as one walk and as the walk token by token, whatever the number of segments: prompts that fill every
    segment, that end inside one and that lie in the first alone; from states that are not zero, twice in a row."""
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(n + vd)
    T, slots = torch.bfloat16, dev([4, 0, 2], torch.int32)
    vectors = {k: dev(v, torch.float32) for k, v in (("a_log", np.linspace(-5.0, 2.0, H)), ("dt_bias", rng.standard_normal(H) - 2.0),
                                                     ("skip", rng.standard_normal(H)))}
    first = dev(rng.standard_normal((6, H * n * vd)), torch.float32)
    states = [first.clone() for _ in range(3)]
    for lengths in ([700, 1, 200], [131, 640, 32]):
        start, _ = packed(lengths)
        N = int(start[-1])
        u, x, B, C = space_rows(rng, T, N, H, G, n, vd)
        z = dev(rng.standard_normal((N, H)), torch.float32)
        count = segments or ops.ssd_segments(3, max(lengths), H, n, vd)
        assert segments or count > 1
        scratch = torch.full((3 * count * H * (n * vd + 1),), 9.0, dtype=torch.float32, device="cuda")
        kw, got = dict(share=H // G, dt_logits=z, **vectors), []
        for i, state in enumerate(states):
            out = torch.full((N, H * vd), 9.0, dtype=torch.float32, device="cuda")
            args = (C, B, x, state, dev(start, torch.int32), slots, out, 3, H, n, vd)
            if i == 0:
                ops.decay_scan(*args, **kw)
            else:
                ops.ssd_prompt(*args, max_new=max(lengths), **kw, **(dict(scratch=scratch, segments=count) if i == 2 else {}))
            got.append(f64(out))
        for other in (1, 2):
            assert np.allclose(got[0], got[other], rtol=2e-4, atol=2e-4)
            assert np.allclose(f64(states[0]), f64(states[other]), rtol=2e-4, atol=2e-4)
    assert np.array_equal(f64(states[2])[[1, 3, 5]], f64(first)[[1, 3, 5]])
    with pytest.raises(ops.KernelError, match="segments"):
        ops.ssd_prompt(*args, max_new=640, segments=2, **kw)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,groups,lead", [(24, 2, 0), (96, 1, 8), (4096, 4, 0), (21, 3, 5), (6000, 1, 0), (10240, 2, 0), (640, 640, 0)])
def test_a_gate_before_a_norm_in_groups(dtype, size, groups, lead):
    """Parts of different loudness: a norm over the row, or over other parts, is far off."""
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(size)
    T, N = torch_dtype(dtype), 6
    o = dev(rng.standard_normal((N, size)) * np.repeat(10.0 ** rng.uniform(-1.5, 1.5, (N, groups)), size // groups, axis=1), torch.float32)
    both, w = dev(rng.standard_normal((N, lead + size)) * 2, T), dev(1 + 0.3 * rng.standard_normal(size), torch.float32)
    out = ops.gate_group_norm(o, both[:, lead:], w, 1e-5, torch.empty((N, size), dtype=T, device="cuda"), groups)
    want = plain.group_rms_norm(f64(o) * plain.silu(f64(both)[:, lead:]), f64(w), 1e-5, groups)
    assert np.allclose(f64(out), want, **close(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("N,hidden,ff,experts,top,shared,limits", [(5, 40, 24, 6, 3, 16, (0.8, 0.3)), (200, 64, 64, 8, 2, 64, (1.0, 2.0)), (33, 96, 32, 1, 1, None, (0.5, None)),
                                                                   (9, 50, 21, 4, 4, 11, (2.0, 0.6)), (70, 128, 160, 16, 5, 96, (1.2, 1.0)), (8, 256, 64, 8, 2, 128, (0.7, 0.4)),
                                                                   (300, 128, 64, 8, 2, 256, (0.7, 0.4)), (1100, 128, 64, 4, 1, 256, (0.7, 0.4))])
def test_clamped_experts_with_biased_logits_and_a_shared_one(dtype, N, hidden, ff, experts, top, shared, limits):
    """The bias decides between experts and is part of the weights; the shared expert is clamped at a limit of its own."""
    import torch
    rng = np.random.default_rng(N + ff)
    T = torch_dtype(dtype)

    def weights(specs):
        out = {}
        for n, s in specs.items():
            if n.endswith("router.b"):
                out[n] = dev(2.0 * rng.permutation(s.shape[0]), torch.float32)
            else:
                out[n] = dev(rng.standard_normal(s.shape) / np.sqrt(s.shape[-1]) * (0.4 if n.endswith("router") else 1.5), T)
        return out
    b = Bound("feed_forward", "routed_experts", {
        "hidden_size": hidden, "intermediate_size": ff, "experts": experts, "top": top, "limit": limits[0], "scoring": "top_logits",
        "router_bias": True, "shared_size": shared, "shared_limit": limits[1], "shared_gate": False, "prefix": "mlp."}, weights, T, N)
    h = dev(rng.standard_normal((N, hidden)), T)
    out = b.part.forward(h, b.ctx)
    mlp = {"expert": {"limit": limits[0]}, "router": {"experts": experts, "top": top}, "shared": {"limit": limits[1]} if shared else None}
    want = plain.experts(f64(h), b.weights, "mlp.", mlp, plain.same if dtype == "float32" else plain.round_bf16)
    tol = 1e-4 if dtype == "float32" else 4e-2
    assert np.allclose(f64(out), want, rtol=tol, atol=tol)
    assert b.ctx.scratch.violations() == []


# ============================================================================ the engine
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("vinozen")
    out = {}
    for i, name in enumerate(sorted(CASES)):
        out[name, "float32"] = make_folder(base, case(name), seed=71 + i, name=name)
        # bfloat16 runs use routers whose choices no rounding can change (see decide_routers)
        out[name, "bfloat16"] = make_folder(base, case(name), seed=71 + i, name=name + "_decided", decided=True)
    return out


def engine_for(folder, dtype, max_tokens, **kw):
    from qwen3_b200 import Engine
    return Engine.from_folder(folder, dtype=dtype, max_tokens=max_tokens, **kw)


def make_requests(cfg, lengths, seed):
    rng = np.random.default_rng(seed)
    return {f"r{i}": random_tokens(rng, n, cfg["vocab"]) for i, n in enumerate(lengths)}


_exact = {}


def oracle(name, weights, toks, cfg=None):
    key = (name, id(weights), tuple(toks))
    if key not in _exact:
        cfg = cfg or case(name)
        exact = plain.logits(toks, weights, cfg)
        rounded = plain.logits(toks, weights, cfg, rnd=plain.round_bf16)
        _exact[key] = (exact, 4.0 * float(np.max(np.abs(rounded - exact))) + 1e-6, float(np.abs(exact).max()))
    return _exact[key]


def check(got, requests, name, weights, dtype, label, cfg=None):
    """32-bit: every row within FP32_TOL.  bfloat16: within four times what rounding does to this very request in the plain
    implementation."""
    for rid, toks in requests.items():
        exact, bf16_tol, scale = oracle(name, weights, toks, cfg)
        tol = FP32_TOL * max(1.0, scale) if dtype == "float32" else bf16_tol
        for p in range(len(toks)):
            if (rid, p) not in got:
                continue
            row = got[(rid, p)]
            assert np.all(np.isfinite(row)), f"{label}: request {rid} position {p}: non-finite logits"
            err = float(np.max(np.abs(row - exact[p])))
            assert err <= tol, f"{label} [{dtype}] case {name}: request {rid} position {p} of {len(toks)}: {err:.3e} > {tol:.3e}"


@pytest.mark.parametrize("name", sorted(CASES))
def test_hidden_rows_after_every_layer(folders, name):
    from qwen3_b200 import StepEntry
    from qwen3_b200.parts.block import settle_any
    folder, weights = folders[name, "float32"]
    cfg = case(name)
    toks = random_tokens(np.random.default_rng(0), 150, cfg["vocab"])
    engine = engine_for(folder, "float32", 192, guard_scratch=True)
    seen = []

    def after_run(run, residual, pending, ctx):
        rows = residual[:ctx.n_tokens].clone()
        settle_any(rows, pending, None, None)
        seen.append(f64(rows))
    engine.model.after_run = after_run
    engine.step([StepEntry(engine.new_sequence(), toks, [0])])
    states = plain.hidden(toks, weights, cfg)
    assert len(seen) == len(states)
    for i, (got, want) in enumerate(zip(seen, states)):
        err = float(np.max(np.abs(got - want)))
        assert err <= 2e-4 * max(1.0, float(np.max(np.abs(want)))), f"case {name}: after layer {i} ({cfg['layers'][i]['type']}): {err:.3e}"
    assert engine.scratch_violations() == []


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,lengths", [("A", [1, 2, 3, 4, 5, 31, 32, 33, 63, 64, 65, 141, 300]), ("B", [1, 63, 64, 65, 127, 128, 129, 260]),
                                          ("C", [1, 2, 31, 64, 127, 128, 129, 192, 193, 450]), ("D", [1, 2, 3, 4, 5, 6, 70, 150])])
def test_whole_requests(folders, name, lengths, dtype):
    folder, weights = folders[name, dtype]
    requests = make_requests(case(name), lengths, seed=1)
    steps, rows = schedules.whole(requests)
    engine = engine_for(folder, dtype, schedules.peak_tokens(steps), guard_scratch=True)
    got = run_steps(engine, steps, rows)
    assert len(got) == sum(lengths)
    check(got, requests, name, weights, dtype, "whole")
    assert engine.cache.pages_held() == 0 and engine.scratch_violations() == []


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,lengths,tail", [("A", [30, 100, 215], 160), ("B", [70, 210], 150), ("C", [230, 420], 260), ("D", [20, 90], 40)])
def test_prompt_then_token_by_token(folders, name, lengths, tail, dtype):
    """The last `tail` tokens one a step: keys pass through every stretch of the biases and over page borders, states and
    convolutions are carried through a long decode (a request shorter than the tail goes token by token from its first token)."""
    folder, weights = folders[name, dtype]
    requests = make_requests(case(name), lengths, seed=2)
    steps, rows = schedules.tail_one_by_one(requests, tail)
    engine = engine_for(folder, dtype, schedules.peak_tokens(steps))
    got = run_steps(engine, steps, rows)
    check(got, requests, name, weights, dtype, "tail one by one")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,length,cuts", [
    ("A", 260, [2, 4, 5, 7, 31, 36, 38, 64, 66, 128, 190, 258]), ("A", 150, list(range(2, 150, 2))),
    ("B", 230, [63, 65, 127, 129, 191, 194]), ("C", 420, [16, 63, 65, 129, 192, 203, 400]), ("D", 100, [2, 4, 6, 8, 10, 12, 50])])
def test_prompts_fed_in_portions(folders, name, length, cuts, dtype):
    """Portions of many sizes, down to two tokens (shorter than the convolutions), that start and end at, before and after the
    edges of pages and chunks."""
    folder, weights = folders[name, dtype]
    requests = make_requests(case(name), [length], seed=3)
    steps, rows = schedules.chunked(requests, {"r0": cuts})
    engine = engine_for(folder, dtype, schedules.peak_tokens(steps))
    got = run_steps(engine, steps, rows)
    assert len(got) == length
    check(got, requests, name, weights, dtype, "portions")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,lengths,prompts,batch", [
    ("A", [13, 130, 9, 90, 76, 45, 128, 3], [5, 100, 1, 69, 41, 40, 39, 3], 3),
    ("B", [140, 70, 200, 66], [130, 1, 64, 63], 2),
    ("C", [300, 110, 9, 260, 210], [199, 104, 1, 133, 103], 3),
    ("D", [30, 7, 50], [8, 7, 1], 3),
])
def test_unequal_batches_one_after_another(folders, name, lengths, prompts, batch, dtype):
    """Requests of different lengths start together and are decoded together; the shorter ones end earlier; the next batch
    takes over their slots, pages and state rows.  Every row must be what the request gives alone."""
    folder, weights = folders[name, dtype]
    requests = make_requests(case(name), lengths, seed=4)
    steps, rows = schedules.batched(requests, dict(zip(requests, prompts)), batch, want_all_prompt=True)
    engine = engine_for(folder, dtype, schedules.peak_tokens(steps), guard_scratch=True)
    got = run_steps(engine, steps, rows)
    check(got, requests, name, weights, dtype, "batches")
    assert engine.cache.pages_held() == 0 and engine.cache.slots.n_free == engine.cache.n_slots
    again = run_steps(engine, steps, rows)                       # the same once more: other slots and pages, same rows
    worst = max(float(np.max(np.abs(got[k] - again[k]))) for k in got)
    assert worst <= (1e-5 if dtype == "float32" else 0.05) * max(1.0, oracle(name, weights, requests["r0"])[2]), worst
    assert engine.scratch_violations() == []


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CASES))
def test_mixed_steps_of_portions_and_single_tokens(folders, name, dtype):
    folder, weights = folders[name, dtype]
    requests = make_requests(case(name), [150, 90, 200], seed=5)
    steps, rows = schedules.mixed(requests, {"r0": 38, "r1": 41, "r2": 1}, {"r0": 1, "r1": 7, "r2": 33})
    engine = engine_for(folder, dtype, schedules.peak_tokens(steps))
    got = run_steps(engine, steps, rows)
    check(got, requests, name=name, weights=weights, dtype=dtype, label="mixed")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_long_decode_and_a_reused_slot_that_starts_from_nothing(folders, dtype):
    from qwen3_b200 import StepEntry
    folder, weights = folders["A", dtype]
    toks = random_tokens(np.random.default_rng(6), 330, case("A")["vocab"])
    engine = engine_for(folder, dtype, 384, n_slots=1)
    for round_ in range(2):
        slot = engine.new_sequence()
        rows = [engine.step([StepEntry(slot, toks[:3], [2])])[0].cpu().numpy()]
        for p in range(3, 330):
            rows.append(engine.step([StepEntry(slot, [toks[p]], [0])])[0].cpu().numpy())
        engine.release(slot)
        check({("r", 2 + i): r for i, r in enumerate(rows)}, {"r": toks}, "A", weights, dtype, "long decode")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["attention", "state space", "shared keys", "bare"])
def test_models_of_one_kind_of_layer(tmp_path, kind, dtype):
    """Only attention (no state at all), only state spaces (no pages at all), one source of keys that every layer reads, no
    feed-forward anywhere: prompt, then token by token."""
    mixers = {"attention": [attention(2, 2, 16, 16, 0.7, 30), attention(4, 1, 32, 32, 0.9, 70, temp=(0.5, 11))],
              "state space": [mamba2(2, 16, 16, 2, 4, 1), mamba2(3, 8, 24, 1, 2, 3)],
              "shared keys": [attention(2, 1, 16, 48, 0.7, 30, temp=(0.2, 9))] + [attention(2, 1, 16, 48, 0.5 + 0.2 * i, 20 * i, kv_from=0) for i in (1, 2, 3)],
              "bare": [mamba2(2, 16, 32, 1, 3, 2), attention(3, 1, 16, 16, 1.0, 50)]}[kind]
    cfg = {"architecture": "Vinozen", "vocab": 80, "width": 40, "embedding": {"scale": 1.5}, "norm": {"eps": 1e-5},
           "token_side": {"dim": 8} if kind != "attention" else None,
           "layers": [layer(m, None if kind == "bare" else (dense(48) if i % 2 else moe_spec(16, 1.0, 4, 2, shared=(24, 0.5)))) for i, m in enumerate(mixers)]}
    folder, weights = make_folder(tmp_path, cfg, seed=12, decided=dtype == "bfloat16")
    requests = make_requests(cfg, [90, 3], seed=13)
    steps, rows = schedules.tail_one_by_one(requests, 40)
    engine = engine_for(folder, dtype, schedules.peak_tokens(steps))
    got = run_steps(engine, steps, rows)
    check(got, requests, "one kind: " + kind, weights, dtype, "one kind", cfg=cfg)
    assert engine.cache.pages_held() == 0 and (len(engine.cache.groups) == 0) == (kind == "state space")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_token_is_found_again_and_a_bias_tells_distances_apart(tmp_path, dtype):
    """Inside a whole model, keys that stand out among hundreds: queries and keys read one channel of the hidden state that one
    token of the vocabulary alone sets.  The last row of the biases is low, so that the marked token weighs less from the
    distance on at which that row begins - and by as much as the plain implementation says."""
    import torch
    import qwen3_b200 as q
    from vinozen_cases import lively_weights
    cfg = {"architecture": "Vinozen", "vocab": 60, "width": 64, "embedding": {"scale": 1.0}, "norm": {"eps": 1e-5}, "token_side": None,
           "layers": [layer(attention(2, 1, 16, 16, 1.0, 100), dense(48)), layer(attention(2, 1, 16, 16, 0.9, 100, kv_from=0), dense(48))]}
    tensors = lively_weights(q.build_model(q.config_from_dict(cfg).plan()).weight_specs(), 31)
    embed, wq, wk = tensors["embed"].float(), tensors["l0.mix.q"].float(), tensors["l0.mix.k"].float()
    embed[:, 5], embed[:, 6] = 0.0, 0.0
    embed[7, 5], embed[8, 6] = 30.0, 30.0                                # token 7 marks its key, token 8 asks for it
    wk[10], wq[10], wq[26] = 0.0, 0.0, 0.0
    wk[10, 5], wq[10, 6], wq[26, 6] = 4.0, 4.0, 4.0
    rel = torch.zeros((16, 2))
    rel[-1] = -3.0
    tensors.update({"embed": embed.to(torch.bfloat16), "l0.mix.q": wq.to(torch.bfloat16), "l0.mix.k": wk.to(torch.bfloat16), "l0.mix.rel": rel.to(torch.bfloat16)})
    folder, weights = make_folder(tmp_path, cfg, seed=0, tensors=tensors)
    filler = [int(t) for t in np.random.default_rng(2).integers(9, 60, 299)]
    edge = next(n for n in range(1000) if plain.bucket(n, 16, 100) == 15)
    requests = {"none": filler + [8]}
    for place in (0, 1, 63, 64, 150, 299 - edge, 300 - edge, 290):
        requests[f"p{place}"] = filler[:place] + [7] + filler[place + 1:] + [8]
    logits = {}
    for steps, rows in (schedules.whole(requests), schedules.tail_one_by_one(requests, 33)):
        engine = engine_for(folder, dtype, schedules.peak_tokens(steps))
        got = run_steps(engine, steps, rows)
        check(got, requests, "far", weights, dtype, "far", cfg=cfg)
        logits = {rid: got[(rid, 299)] for rid in requests}
    for rid in logits:
        assert rid == "none" or float(np.max(np.abs(logits[rid] - logits["none"]))) > 0.1, rid      # it shows


@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_greedy_generation_through_the_entry_point(folders, name):
    import qwen3_b200 as q
    folder, weights = folders[name, "float32"]
    cfg = case(name)
    rng = np.random.default_rng(7)
    prompts = [random_tokens(rng, n, cfg["vocab"]) for n in (5, 38, 1, 70)]

    def greedy(prompt, n):
        toks = list(prompt)
        for _ in range(n):
            toks.append(int(np.argmax(plain.logits(toks, weights, cfg)[-1])))
        return toks[len(prompt):]
    engine = engine_for(folder, "float32", 64 * 8)
    got = q.generate_token_ids(engine, prompts, q.SamplingParams.greedy(), q.GenerationOptions(max_new_tokens=10))
    for p, r in zip(prompts, got):
        assert r.token_ids == greedy(p, 10) and r.stop_reason == q.MAX_NEW_TOKENS
    assert engine.cache.pages_held() == 0
    small = engine_for(folder, "float32", 64 * 4, n_slots=2)      # fewer slots than requests: one batch after another
    again = q.generate_token_ids(small, prompts, q.SamplingParams.greedy(), q.GenerationOptions(max_new_tokens=10))
    assert [r.token_ids for r in again] == [r.token_ids for r in got]


def test_the_command_line_generates_from_token_ids(folders):
    """bin/qwen3_chat on a Vinozen folder: the model class comes from config.json; greedy sampling through the scheduler."""
    import subprocess
    import sys
    folder, weights = folders["A", "float32"]
    cfg = case("A")
    prompts = [[7, 8, 9, 150, 2], [100, 3]]
    out = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "qwen3_chat"), folder, "--greedy", "--dtype", "float32",
                          "--max-new-tokens", "9", "--max-context", "64", "--tokens", "7,8,9,150,2", "--tokens", "100 3"],
                         capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    lines = [l for l in out.stdout.strip().splitlines() if l and l[0].isdigit()]
    assert len(lines) == 2
    for p, line in zip(prompts, lines):
        toks = list(p)
        for _ in range(9):
            toks.append(int(np.argmax(plain.logits(toks, weights, cfg)[-1])))
        assert [int(t) for t in line.split("#")[0].strip().split(",")] == toks[len(p):]


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_from_the_command_line(tmp_path, folders, dtype, monkeypatch):
    from test_trace_run_gpu import replay
    unpadded = schedules.peak_tokens
    monkeypatch.setattr(schedules, "peak_tokens", lambda steps, page=64: unpadded(steps, 1))
    folder, weights = folders["A", dtype]
    cfg = case("A")
    requests = make_requests(cfg, [75, 1, 130], seed=8)
    w_steps, w_rows = schedules.whole(requests)
    b_steps, b_rows = schedules.batched(requests, {"r0": 40, "r1": 1, "r2": 81}, 3)
    steps, rows = [], []
    for part_steps, part_rows in ((w_steps, w_rows), (b_steps, b_rows)):
        for s, r in zip(part_steps, part_rows):
            steps.append(dict(s, step=len(steps)))
            rows.append([(f"{len(steps)}:{rid}", rid, p) for rid, p in r])
    got = replay(folder, dtype, steps, [[(tag, p) for tag, _, p in r] for r in rows], str(tmp_path / "out"), cfg["vocab"])
    for r in rows:
        for tag, rid, p in r:
            exact, bf16_tol, scale = oracle("A", weights, requests[rid])
            err = float(np.max(np.abs(got[(tag, p)] - exact[p])))
            assert err <= (FP32_TOL * max(1.0, scale) if dtype == "float32" else bf16_tol), (tag, p, err)
