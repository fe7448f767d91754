"""Vogerax on the GPU against the plain implementation (tests/plain/vogerax_plain.py): every mechanism alone,
then the engine under every way of cutting requests into steps, in 32-bit and in bfloat16."""
import os

import numpy as np
import pytest

import schedules
from plain import vogerax_plain as plain
from test_engine_gpu import run_steps
from vogerax_cases import CASES, attention, case, dense, layer, make_folder, parallel, random_tokens, retention, rotated
from vogerax_cases import moe as moe_spec

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


# ============================================================================ mechanisms, one at a time
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,post,pre", [(64, 4, 4), (64, 1, 8), (50, 5, 5), (48, 12, 3), (2048, 2, 2), (3072, 8, 1), (12, 12, 12), (6000, 3, 2),
                                           (9000, 4, 4), (40, 40, 1), (16384, 2, 2)])
def test_norms_in_groups_around_the_residual_sum(dtype, size, post, pre):
    """Both norms of a pass in groups, or only one; parts of different loudness, so that a norm over the whole row, or over
    the wrong parts, is far off."""
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(size + post)
    T, N = torch_dtype(dtype), 7

    def rows():
        return rng.standard_normal((N, size)) * np.repeat(10.0 ** rng.uniform(-1.5, 1.5, (N, post * pre if size % (post * pre) == 0 else 1)),
                                                          size // (post * pre) if size % (post * pre) == 0 else size, axis=1)
    stream, branch = dev(rows(), torch.float32), dev(rows(), T)
    w_post, w_pre = (dev(1 + 0.3 * rng.standard_normal(size), torch.float32) for _ in range(2))
    for use_branch, use_out in ((True, True), (True, False), (False, True)):
        x, out = stream.clone(), torch.full((N, size), 9.0, dtype=T, device="cuda")
        ops.sandwich_norm(x, branch if use_branch else None, w_post if use_branch else None, 1e-4, w_pre if use_out else None, 1e-5,
                          out if use_out else None, groups_post=post, groups_pre=pre)
        want = f64(stream) + (plain.group_norm(f64(branch), f64(w_post), 1e-4, post) if use_branch else 0.0)
        assert np.allclose(f64(x), want, rtol=1e-5, atol=1e-4)
        if use_out:
            assert np.allclose(f64(out), plain.group_norm(want, f64(w_pre), 1e-5, pre), **close(dtype))
    idx = dev([3, 0, 6, 3], torch.int32)
    picked = torch.empty((4, size), dtype=T, device="cuda")
    ops.gather_rows_norm(stream, idx, w_pre, 1e-5, picked, groups=pre)
    assert np.allclose(f64(picked), plain.group_norm(f64(stream), f64(w_pre), 1e-5, pre)[[3, 0, 6, 3]], **close(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [7, 64, 320, 2048, 4100, 9000])
def test_two_normed_branches_are_summed(dtype, size):
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(size)
    T, N = torch_dtype(dtype), 5
    a, b = dev(rng.standard_normal((N, size)) * 30, T), dev(rng.standard_normal((N, size)) * 0.01, T)
    wa, wb = (dev(1 + 0.3 * rng.standard_normal(size), torch.float32) for _ in range(2))
    out = ops.normed_sum(a, b, wa, wb, 0.5, -0.75, 1e-5, torch.empty_like(a))
    want = 0.5 * plain.rms_norm(f64(a), f64(wa), 1e-5) - 0.75 * plain.rms_norm(f64(b), f64(wb), 1e-5)
    assert np.allclose(f64(out), want, **close(dtype))


def scattered_pages(rng, lengths, heads, width, T, columns=6):
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
    return np.stack([p[table[s, j // PAGE], :, j % PAGE] for j in range(n)]) if n else np.zeros((0,) + p.shape[1:2] + p.shape[3:])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("lengths", [[3, 1, 9], [90, 1, 70]])          # few tokens: a warp a head; many: 16-byte packets where sizes allow
@pytest.mark.parametrize("H,G,d,vd,dims,tied,norm,turned,gate", [
    (4, 2, 16, 16, 8, True, False, False, False), (2, 1, 64, 64, 16, True, False, False, False), (3, 3, 11, 11, 10, True, False, False, False),
    (2, 2, 32, 32, 32, True, True, False, True), (2, 2, 16, 16, 0, True, False, False, False),
    (4, 2, 16, 24, 8, False, True, True, True), (2, 2, 64, 64, 48, False, True, True, True), (1, 1, 128, 128, 64, False, True, True, False),
    (2, 1, 5, 10, 4, False, True, True, True), (2, 1, 32, 32, 0, False, False, True, True)])
def test_rows_are_prepared_and_cached(dtype, lengths, H, G, d, vd, dims, tied, norm, turned, gate):
    """Values that are the projected keys (before norm and rotation), scaled rotations of a part of the head with a magnitude,
    values rotated by their own position, rows with further columns behind the values."""
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(d * 10 + H + len(lengths))
    T, eps = torch_dtype(dtype), 1e-5
    pos0 = [0, 100, 7]
    start, seq = packed(lengths)
    pos = np.concatenate([np.arange(p, p + n) for p, n in zip(pos0, lengths)]).astype(np.int32)
    N, columns = len(pos), (H + G) * d + (0 if tied else G * vd)
    rows = dev(rng.standard_normal((N, columns + (H * vd if gate else 0))), T)
    table, k_pages = scattered_pages(rng, [p + n for p, n in zip(pos0, lengths)], G, d, T)
    v_pages = torch.zeros(k_pages.shape[:-1] + (vd,), dtype=T, device="cuda")
    freq, magnitude = plain.yarn(300.0, dims, {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 0.5}) if dims else (None, 1.0)
    v_freq = plain.plain_frequencies(300.0, vd)

    def tables(f, m):
        a = np.arange(200)[:, None] * f[None, :]
        return dev(m * np.cos(a), torch.float32), dev(m * np.sin(a), torch.float32)
    cos, sin = tables(freq, magnitude) if dims else (None, None)
    v_cos, v_sin = tables(v_freq, 1.0) if turned else (None, None)
    qw, kw = ((dev(1 + 0.3 * rng.standard_normal(d), torch.float32) for _ in range(2)) if norm else (None, None))
    q = torch.empty((N, H * d), dtype=T, device="cuda")
    ops.qkv_prepare(rows, q, k_pages, v_pages, qw, kw, cos, sin, dev(seq, torch.int32), dev(pos, torch.int32), dev(table, torch.int32),
                    N, H, G, d, eps, value_dim=vd, tied_values=tied, norm_once=True, value_cos=v_cos, value_sin=v_sin)
    x = f64(rows)
    qs, ks = x[:, :H * d].reshape(N, H, d), x[:, H * d:(H + G) * d].reshape(N, G, d)
    vs = ks if tied else x[:, (H + G) * d:columns].reshape(N, G, vd)
    if norm:
        qs, ks = plain.rms_norm(qs, f64(qw), eps), plain.rms_norm(ks, f64(kw), eps)
    if dims:
        qs, ks = plain.rotary(qs, pos, freq, magnitude), plain.rotary(ks, pos, freq, magnitude)
    if turned:
        vs = plain.rotary(vs, pos, v_freq)
    tol = dict(rtol=1e-5, atol=3e-5) if dtype == "float32" else dict(rtol=2 ** -8, atol=1e-5)      # one rounding
    assert np.allclose(f64(q).reshape(N, H, d), qs, **tol)
    for s, (p, n) in enumerate(zip(pos0, lengths)):
        assert np.allclose(read_pages(k_pages, table, s, p + n)[p:], ks[start[s]:start[s + 1]], **tol)
        assert np.allclose(read_pages(v_pages, table, s, p + n)[p:], vs[start[s]:start[s + 1]], **tol)
        assert np.all(read_pages(k_pages, table, s, p + n)[:p] == 0.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,vd,turn,gate", [(3, 10, True, True), (2, 64, True, True), (4, 128, True, False), (2, 24, False, True), (1, 2, True, True),
                                                (2, 256, True, True)])
def test_heads_are_turned_back_and_gated(dtype, heads, vd, turn, gate):
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(vd)
    T, N = torch_dtype(dtype), 19
    pos = rng.integers(0, 500, N)
    freq = plain.plain_frequencies(700.0, vd)
    a = np.arange(500)[:, None] * freq[None, :]
    x = dev(rng.standard_normal((N, heads * vd)), T)
    both = dev(rng.standard_normal((N, 8 + heads * vd)) * 2, T)
    want = f64(x).reshape(N, heads, vd)
    if turn:
        want = plain.rotary(want, pos, freq, sign=-1.0)
    want = want.reshape(N, -1) * (plain.sigmoid(f64(both)[:, 8:]) if gate else 1.0)
    got = ops.turn_back_gate(x, dev(np.cos(a), torch.float32) if turn else None, dev(np.sin(a), torch.float32) if turn else None,
                             dev(pos, torch.int32), both[:, 8:] if gate else None, heads, vd)
    assert np.allclose(f64(got), want, **close(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,d,vd,dims", [(2, 8, 12, 8), (1, 16, 48, 0), (2, 128, 128, 128), (4, 16, 32, 6), (3, 5, 9, 4), (2, 64, 24, 16), (1, 256, 64, 2)])
def test_retention_over_unequal_sequences_and_from_its_state(dtype, heads, d, vd, dims):
    """Whole prompts in chunks, portions and single tokens on slots in no particular order; the state is carried in columns
    of a wider row, as a mixer beside another mixer holds it; decays from 0 to 1; every form of the kernel."""
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(heads * 1000 + d + vd)
    T, k_scale = torch_dtype(dtype), d ** -0.5
    freq = plain.plain_frequencies(90.0, dims) if dims else None
    angle = np.arange(400)[:, None] * freq[None, :] if dims else None
    cos, sin = (dev(np.cos(angle), torch.float32), dev(np.sin(angle), torch.float32)) if dims else (None, None)
    decay = np.array([0.97, 0.0, 1.0, 0.6])[:heads]
    slots, n_slots, before, after, cells = [4, 0, 5, 2], 7, 3, 2, heads * d * vd
    whole = torch.zeros((n_slots + 1, before + cells + after), dtype=torch.float32, device="cuda")
    whole[:, :before], whole[:, before + cells:] = 7.0, -7.0
    state = whole[:, before:before + cells]
    S, length = {s: np.zeros((heads, d, vd)) for s in slots}, {s: 0 for s in slots}
    tol = dict(rtol=3e-4, atol=3e-4) if dtype == "float32" else dict(rtol=2e-3, atol=2e-3)      # nothing is rounded on the way
    for lengths, chunked in (([1, 70, 2, 33], True), ([3, 1, 0, 2], False), ([40, 32, 31, 1], True), ([1, 1, 1, 1], False)):
        live = [(s, n) for s, n in zip(slots, lengths) if n > 0]
        start, _ = packed([n for _, n in live])
        N = int(start[-1])
        pos = np.concatenate([np.arange(length[s], length[s] + n) for s, n in live])
        proj = dev(rng.standard_normal((N, 2 * heads * (d + vd))) * 0.7, T)
        out = torch.full((N, heads * vd), 9.0, dtype=torch.float32, device="cuda")
        ops.lightning_attention(proj, state, dev(decay, torch.float32), dev(start, torch.int32), dev([s for s, _ in live], torch.int32), out,
                                len(live), heads, d, vd, chunked and ops.lightning_chunks_fit(d, vd), silu=False, k_scale=k_scale, cos=cos,
                                sin=sin, token_pos=dev(pos, torch.int32))
        x = f64(proj)
        q, k = x[:, :heads * d].reshape(N, heads, d), x[:, heads * d:2 * heads * d].reshape(N, heads, d)
        v = x[:, 2 * heads * d:2 * heads * d + heads * vd].reshape(N, heads, vd)
        if dims:
            q, k = plain.rotary(q, pos, freq), plain.rotary(k, pos, freq)
        got = f64(out).reshape(N, heads, vd)
        for i, (slot, n) in enumerate(live):
            for t in range(start[i], start[i + 1]):
                for a in range(heads):
                    S[slot][a] = decay[a] * S[slot][a] + np.outer(k[t, a] * k_scale, v[t, a])
                    assert np.allclose(got[t, a], S[slot][a].T @ q[t, a], **tol), (lengths, slot, t - start[i], a)
            length[slot] += n
    final = f64(whole)
    for slot in slots:
        assert np.allclose(final[slot, before:-after].reshape(heads, d, vd), S[slot], **tol)
    assert np.all(final[:, :before] == 7.0) and np.all(final[:, -after:] == -7.0) and np.all(final[[1, 3, 6, 7], before:-after] == 0.0)


@pytest.mark.parametrize("heads,d,vd,dims,silu", [(2, 16, 24, 8, False), (1, 64, 128, 64, False), (3, 128, 64, 0, True)])
@pytest.mark.parametrize("segments", [None, 2, 3, 7])
def test_long_prompts_walked_in_segments_side_by_side(heads, d, vd, dims, silu, segments):
    """The same numbers as one walk, whatever the number of segments: prompts that fill every segment, that end inside one and
    that lie in the first alone; from states that are not zero, twice in a row."""
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(d + vd)
    T, decay = torch.bfloat16, dev(np.array([0.999, 0.9, 0.0])[:heads], torch.float32)
    angle = np.arange(2000)[:, None] * plain.plain_frequencies(90.0, dims)[None, :] if dims else None
    kw = dict(silu=silu, k_scale=d ** -0.5)
    if dims:
        kw.update(cos=dev(np.cos(angle), torch.float32), sin=dev(np.sin(angle), torch.float32))
    first = dev(rng.standard_normal((6, heads * d * vd)), torch.float32)
    states, outs = [first.clone(), first.clone()], []
    at = {s: 0 for s in (4, 0, 2)}
    for lengths in ([700, 1, 200], [131, 640, 32]):
        start, _ = packed(lengths)
        N = int(start[-1])
        pos = np.concatenate([np.arange(at[s], at[s] + n) for s, n in zip((4, 0, 2), lengths)])
        proj = dev(rng.standard_normal((N, 2 * heads * (d + vd))) * 0.7, T)
        count = segments or ops.lightning_segments(T, 3, max(lengths), heads, d, vd)
        assert segments or count > 1
        scratch = torch.full((3 * count * heads * d * vd,), 9.0, dtype=torch.float32, device="cuda")
        got = []
        for state, more in zip(states, (dict(), dict(scratch=scratch, max_new=max(lengths), segments=count))):
            out = torch.full((N, heads * vd), 9.0, dtype=torch.float32, device="cuda")
            ops.lightning_attention(proj, state, decay, dev(start, torch.int32), dev([4, 0, 2], torch.int32), out, 3, heads, d, vd, True,
                                    token_pos=dev(pos, torch.int32), **kw, **more)
            got.append(f64(out))
        assert np.allclose(got[0], got[1], rtol=1e-4, atol=1e-4)
        assert np.allclose(f64(states[0]), f64(states[1]), rtol=1e-4, atol=1e-4)
        for s, n in zip((4, 0, 2), lengths):
            at[s] += n
    assert np.array_equal(f64(states[1])[[1, 3, 5]], f64(first)[[1, 3, 5]])
    with pytest.raises(ops.KernelError, match="segments"):
        ops.lightning_attention(proj, states[0], decay, dev(start, torch.int32), dev([4, 0, 2], torch.int32), out, 3, heads, d, vd, True,
                                token_pos=dev(pos, torch.int32), segments=2, **kw)


@pytest.mark.parametrize("dtype", DTYPES)
def test_retention_s_heads_are_normed_without_a_weight_and_gated(dtype):
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(8)
    T, N, heads, vd = torch_dtype(dtype), 11, 3, 20
    o = dev(rng.standard_normal((N, heads * vd)) * np.repeat([0.01, 1.0, 50.0], vd), torch.float32)
    gate = dev(rng.standard_normal((N, heads * vd)) * 2, T)
    out = ops.head_gated_norm(o, None, gate, 1e-5, torch.empty((N, heads * vd), dtype=T, device="cuda"), heads, vd, act="silu")
    want = plain.rms_unit(f64(o).reshape(N, heads, vd), 1e-5).reshape(N, -1) * plain.silu(f64(gate))
    assert np.allclose(f64(out), want, **close(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("N,hidden,ff,experts,top,tiles", [(5, 40, 24, 6, 3, None), (200, 64, 64, 8, 2, True), (200, 64, 64, 8, 2, False), (33, 96, 32, 1, 1, True),
                                                           (9, 50, 21, 4, 4, None), (70, 128, 160, 16, 5, True)])
def test_squared_relu_experts_with_a_shared_one(dtype, N, hidden, ff, experts, top, tiles, monkeypatch):
    """The whole routed feed-forward: choice by plain softmax scores, weights not renormalised, experts without a gate, a
    shared expert added as it is; `tiles`: the tensor-core tiles on or off (bfloat16)."""
    import torch
    from qwen3_b200.csrc import ops
    from qwen3_b200.engine.context import Scratch
    from qwen3_b200.parts import build_part
    from qwen3_b200.config import PartSpec
    if tiles is not None:
        monkeypatch.setattr(ops, "moe_tensor_cores", tiles)
    rng = np.random.default_rng(N + ff)
    T = torch_dtype(dtype)
    part = build_part("feed_forward", PartSpec("routed_experts", {
        "hidden_size": hidden, "intermediate_size": ff, "experts": experts, "top": top, "expert_activation": "relu2",
        "shared_size": ff + 3, "shared_gate": False, "correction": False, "prefix": "mlp."}))
    w = {n: dev(rng.standard_normal(s.shape) / np.sqrt(s.shape[-1]) * (3.0 if n.endswith("router") else 1.0), T)
         for n, s in part.weight_specs("l0.").items()}
    weights = {n[len("l0."):]: f64(t) for n, t in w.items()}
    assert sorted(weights) == sorted(["mlp.router", "mlp.shared.up", "mlp.shared.down"] + [f"mlp.e{e}.{m}" for e in range(experts) for m in ("up", "down")])
    from qwen3_b200.weights.upload import TensorDict
    part.bind(TensorDict(dict(w), part.weight_specs("l0."), T, torch.device("cuda"), lambda n: None), "l0.", T, torch.device("cuda"))

    class Ctx:
        n_tokens, scratch = N, Scratch("cuda", guard=True)
    Ctx.dtype = T
    h = dev(rng.standard_normal((N, hidden)), T)
    out = part.forward(h, Ctx)
    mlp = {"router": {"experts": experts, "top": top}, "shared": {"ff": ff + 3}}
    rnd = plain.same if dtype == "float32" else plain.round_bf16
    want = plain.mixture(f64(h), weights, "mlp.", mlp, rnd)
    assert np.allclose(f64(out), want, rtol=1e-4 if dtype == "float32" else 3e-2, atol=1e-4 if dtype == "float32" else 3e-2)
    assert Ctx.scratch.violations() == []


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,hidden,ff", [(1, 64, 48), (5, 256, 512), (8, 40, 30), (100, 128, 264), (300, 96, 512), (700, 512, 1024)])
def test_dense_squared_relu_feed_forward(dtype, rows, hidden, ff):
    """Few rows, a batch's and a prompt's: the product's forms with the activation in or after them."""
    import torch
    from qwen3_b200.config import PartSpec
    from qwen3_b200.engine.context import Scratch
    from qwen3_b200.parts import build_part
    from qwen3_b200.weights.upload import TensorDict
    rng = np.random.default_rng(rows)
    T = torch_dtype(dtype)
    part = build_part("feed_forward", PartSpec("dense_mlp", {"hidden_size": hidden, "intermediate_size": ff, "activation": "relu2",
                                                             "names": {"up": "up", "down": "down"}}))
    w = {n: dev(rng.standard_normal(s.shape) / np.sqrt(s.shape[-1]), T) for n, s in part.weight_specs("").items()}
    weights = {n: f64(t) for n, t in w.items()}
    part.bind(TensorDict(dict(w), part.weight_specs(""), T, torch.device("cuda"), lambda n: None), "", T, torch.device("cuda"))

    class Ctx:
        n_tokens, scratch = rows, Scratch("cuda", guard=True)
    Ctx.dtype = T
    h = dev(rng.standard_normal((rows, hidden)), T)
    want = plain.relu_squared(f64(h) @ weights["up"].T) @ weights["down"].T
    got = f64(part.forward(h, Ctx))
    assert np.allclose(got, want, **(dict(rtol=1e-4, atol=1e-4) if dtype == "float32" else dict(rtol=3e-2, atol=3e-2)))
    assert Ctx.scratch.violations() == []


@pytest.mark.parametrize("form,M,N,K,splits", [("skinny", 1, 48, 64, 0), ("skinny", 8, 4800, 256, 0), ("skinny", 40, 130, 72, 0), ("mid", 9, 100, 256, 0),
                                               ("mid", 100, 520, 2048, 4), ("mid", 300, 257, 128, 1), ("pair", 300, 512, 256, 1), ("pair", 513, 264, 512, 2),
                                               ("pair", 129, 77, 192, 3)])
def test_products_with_the_square_of_relu_in_their_epilogue(form, M, N, K, splits):
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(M + N)
    x, w = dev(rng.standard_normal((M, K)), torch.bfloat16), dev(rng.standard_normal((N, K)) / np.sqrt(K), torch.bfloat16)
    out = ops.gemm_relu2(x, w, torch.full((M, N), -1.0, dtype=torch.bfloat16, device="cuda"), form, splits=splits)
    want = plain.relu_squared(f64(x) @ f64(w).T)
    assert np.allclose(f64(out), want, rtol=2 ** -7, atol=1e-4) and (want == 0.0).any()
    assert ops.tcgen05_status(torch.device("cuda")) == 0
    with pytest.raises(ops.KernelError):
        ops.gemm_relu2(x, w, out, "other")


# ---------------------------------------------------------------- pooled blocks
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("G,d,vd,size", [(2, 16, 16, 5), (1, 64, 64, 16), (3, 11, 7, 3), (1, 128, 128, 1), (2, 8, 8, 64), (1, 8, 24, 100)])
def test_blocks_are_pooled_when_their_last_token_comes(dtype, G, d, vd, size):
    """Steps of many sizes over scattered pages: every block has the means of its cached keys and values after the step that
    brought its last token, whatever steps brought the others; blocks that are not whole are not written."""
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(size)
    T, totals = torch_dtype(dtype), [230, 70, 131]
    table, k_pages = scattered_pages(rng, totals, G, d, T)
    v_pages = torch.zeros(k_pages.shape[:-1] + (vd,), dtype=T, device="cuda")
    pool_table, pool_k = scattered_pages(rng, [max(n // size, 1) for n in totals], G, d, T)
    pool_v = torch.zeros(pool_k.shape[:-1] + (vd,), dtype=T, device="cuda")
    pool = ops.Pool(pool_k, pool_v, dev(pool_table, torch.int32), size)
    keys, values = [rng.standard_normal((n, G, d)) for n in totals], [rng.standard_normal((n, G, vd)) for n in totals]
    done = [0, 0, 0]
    for new in ([1, 64, 4], [4, 1, 1], [1, 1, 1], [59, 2, 60], [1, 1, 1], [2, 1, 63], [162, 0, 1]):
        live = [s for s in range(3) if new[s] > 0]
        for s in live:
            for j in range(done[s], done[s] + new[s]):
                k_pages[table[s, j // PAGE], :, j % PAGE] = dev(keys[s][j], T)
                v_pages[table[s, j // PAGE], :, j % PAGE] = dev(values[s][j], T)
        start, _ = packed([new[s] for s in live])
        rows = dev(table[live], torch.int32)
        ops.pool_blocks(k_pages, v_pages, rows, ops.Pool(pool_k, pool_v, dev(pool_table[live], torch.int32), size), dev(start, torch.int32),
                        dev([done[s] for s in live], torch.int32), len(live), max(new))
        for s in live:
            done[s] += new[s]
        for s in range(3):
            n = done[s] // size
            k, v = read_pages(k_pages, table, s, done[s]), read_pages(v_pages, table, s, done[s])
            tol = dict(rtol=1e-5, atol=1e-6) if dtype == "float32" else dict(rtol=2 ** -8, atol=1e-6)
            assert np.allclose(read_pages(pool_k, pool_table, s, n), plain.pooled_blocks(k, size), **tol), (new, s)
            assert np.allclose(read_pages(pool_v, pool_table, s, n), plain.pooled_blocks(v, size), **tol), (new, s)
            rest = read_pages(pool_k, pool_table, s, min(max(totals[s] // size, 1), n + 3))[n:]
            assert np.all(rest == 0.0)
    assert pool.size == size


LENGTHS = [400, 70, 1, 131]
WHERE = ["window_in", "window_out", "pool_in", "pool_out", "pool_far", "self"]


def planted(rng, H, G, d, window, size, where):
    """Sequences in which, for every query, one place has a score that towers over the others if it is seen: the window's first
    token, the token before it, the last block that is seen, the first that is not yet, an early block, the token itself.
    A block is marked in all its tokens, so that its mean carries the mark."""
    seqs = []
    for n in LENGTHS:
        q, k = rng.standard_normal((n, H, d)) * 0.3, rng.standard_normal((n, G, d)) * 0.3
        v = rng.standard_normal((n, G, d))
        for p in range(n):
            lo = max(p - window + 1, 0)
            blocks = lo // size
            if where == "window_in":
                tokens = [lo]
            elif where == "window_out":
                tokens = [lo - 1] if lo > 0 else []
            elif where == "self":
                tokens = [p]
            else:
                b = {"pool_in": blocks - 1, "pool_out": blocks, "pool_far": blocks // 3}[where]
                tokens = [j for j in range(b * size, (b + 1) * size) if 0 <= j < n] if b >= 0 else []
            if not tokens or rng.random() > 0.5:        # some queries without a mark of their own
                continue
            mark = rng.standard_normal(d)
            mark /= np.linalg.norm(mark)
            k[tokens] += 5.0 * mark
            q[p] += 6.0 * mark
        seqs.append((q, k, v))
    return seqs


def pooled_pages(rng, T, seqs, G, d, size):
    """The sequences' keys and values in scattered pages, and their pooled blocks made by the kernel."""
    import torch
    from qwen3_b200.csrc import ops
    table, k_pages = scattered_pages(rng, LENGTHS, G, d, T, columns=7)
    v_pages = torch.zeros_like(k_pages)
    for s, (q, k, v) in enumerate(seqs):
        for pg in range(-(-LENGTHS[s] // PAGE)):
            rows = slice(pg * PAGE, min(LENGTHS[s], (pg + 1) * PAGE))
            k_pages[table[s, pg], :, :rows.stop - rows.start] = dev(k[rows], T).transpose(0, 1)
            v_pages[table[s, pg], :, :rows.stop - rows.start] = dev(v[rows], T).transpose(0, 1)
    pool_table, pool_k = scattered_pages(rng, [max(n // size, 1) for n in LENGTHS], G, d, T, columns=7)
    pool = ops.Pool(pool_k, torch.zeros_like(pool_k), dev(pool_table, torch.int32), size)
    start, _ = packed(LENGTHS)
    ops.pool_blocks(k_pages, v_pages, dev(table, torch.int32), pool, dev(start, torch.int32), dev([0] * 4, torch.int32), 4, max(LENGTHS))
    return k_pages, v_pages, table, pool, pool_table


def without_unseen(table, take, window):
    """The page table as the cache leaves it: pages that hold no token that a query of `take` sees are given back."""
    gone = table.copy()
    for s in range(len(LENGTHS)):
        first = min(p for t, ps in take if t == s for p in ps)
        for pg in range(max(first - window + 1, 0) // PAGE):
            gone[s, pg] = -1
    return gone


def pooled_oracle(seqs, T, window, size, scale, rnd):
    """Per sequence [n, H, d]."""
    out = []
    for q, k, v in seqs:
        q, k, v = (f64(dev(a, T)) for a in (q, k, v))
        n = q.shape[0]
        tokens, blocks = plain.visible(n, window, size)
        keys, values = np.concatenate([k, rnd(plain.pooled_blocks(k, size))]), np.concatenate([v, rnd(plain.pooled_blocks(v, size))])
        out.append(plain.softmax_attention(q, keys, values, scale, np.concatenate([tokens, blocks], axis=1)))
    return out


def queries(seqs, take):
    return np.concatenate([seqs[s][0][p] for s, p in take])


TAKE = [(0, list(range(400))), (1, list(range(40, 70))), (2, [0]), (3, [130])]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,window,size", [(4, 2, 16, 37, 5), (2, 1, 64, 70, 1), (3, 3, 5, 1, 2), (2, 2, 32, 64, 64), (4, 1, 64, 130, 3), (1, 1, 8, 20, 33)])
@pytest.mark.parametrize("where", WHERE)
def test_attention_sees_the_window_and_the_blocks_before_it(dtype, H, G, d, window, size, where):
    """The general kernel over pages, one place made to stand out; whole prompts, a portion, single tokens; pages that no
    query sees are gone."""
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(d * 100 + window)
    T = torch_dtype(dtype)
    seqs = planted(rng, H, G, d, window, size, where)
    k_pages, v_pages, table, pool, _ = pooled_pages(rng, T, seqs, G, d, size)
    want = pooled_oracle(seqs, T, window, size, 0.5, plain.same if dtype == "float32" else plain.round_bf16)
    seq = np.concatenate([np.full(len(p), s) for s, p in TAKE]).astype(np.int32)
    pos = np.concatenate([p for _, p in TAKE]).astype(np.int32)
    N = len(pos)
    out = torch.empty((N, H * d), dtype=T, device="cuda")
    ops.attention_generic(dev(queries(seqs, TAKE).reshape(N, H * d), T), k_pages, v_pages, out, dev(seq, torch.int32), dev(pos, torch.int32),
                          dev(without_unseen(table, TAKE, window), torch.int32), N, H, G, d, 0.5, window=window, pool=pool)
    got = f64(out).reshape(N, H, d)
    for row in range(N):
        assert np.allclose(got[row], want[seq[row]][pos[row]], atol=3e-5 if dtype == "float32" else 3e-2), (where, seq[row], pos[row])


@pytest.mark.parametrize("H,G,d,window,size", [(4, 2, 16, 37, 5), (2, 1, 64, 70, 1), (2, 2, 32, 64, 64), (4, 1, 64, 130, 3), (16, 1, 16, 1, 2), (2, 2, 128, 200, 7),
                                               (2, 1, 64, 20, 33)])
@pytest.mark.parametrize("where", WHERE)
def test_tiled_attention_walks_the_blocks_before_the_window_s_pages(H, G, d, window, size, where):
    """The tensor-core kernels of the bfloat16 path: prompts and portions in tiles of 64 rows, single tokens with the pages
    split over 1, 2 and 5 blocks."""
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(d * 100 + window + 1)
    T = torch.bfloat16
    seqs = planted(rng, H, G, d, window, size, where)
    k_pages, v_pages, table, pool, pool_table = pooled_pages(rng, T, seqs, G, d, size)
    want = pooled_oracle(seqs, T, window, size, 0.5, plain.round_bf16)
    start, seq = packed([len(p) for _, p in TAKE])
    pos = np.concatenate([p for _, p in TAKE])
    N = len(pos)
    out = torch.empty((N, H * d), dtype=T, device="cuda")
    ops.attention_capped_prefill(dev(queries(seqs, TAKE).reshape(N, H * d), T), k_pages, v_pages, out, dev(start, torch.int32),
                                 dev([p[0] for _, p in TAKE], torch.int32), dev(without_unseen(table, TAKE, window), torch.int32), len(TAKE),
                                 max(LENGTHS), H, G, d, d, 0.5, 0.0, None, False, window=window, pool=pool)
    got = f64(out).reshape(N, H, d)
    for row in range(N):
        assert np.allclose(got[row], want[seq[row]][pos[row]], atol=3e-2), (where, seq[row], pos[row])
    for last in ([399, 69, 0, 130], [200, 63, 0, 64], [window, size - 1 if size <= 70 else 0, 0, window + size - 1 if window + size < 131 else 5]):
        take = [(s, [p]) for s, p in enumerate(last)]
        for splits in (1, 2, 5):
            scratch = torch.empty(4 * H * splits * (d + 2), dtype=torch.float32, device="cuda")
            out = torch.empty((4, H * d), dtype=T, device="cuda")
            ops.attention_capped_decode(dev(queries(seqs, take).reshape(4, H * d), T), k_pages, v_pages, out, scratch,
                                        dev(np.arange(4), torch.int32), dev(last, torch.int32), dev(without_unseen(table, take, window), torch.int32),
                                        4, H, G, d, d, 0.5, 0.0, None, False, splits, window=window, pool=pool)
            got = f64(out).reshape(4, H, d)
            for s, p in enumerate(last):
                assert np.allclose(got[s], want[s][p], atol=3e-2), (where, s, p, splits)


@pytest.mark.parametrize("H,G,d,size,window", [(4, 2, 16, 5, 9), (2, 1, 64, 16, 20), (2, 2, 128, 1, 3), (1, 1, 32, 70, 70)])
def test_the_split_decode_pools_a_block_that_its_token_completes(H, G, d, size, window):
    """Token by token over a page's worth of blocks: after every step the pool holds exactly the whole blocks, and the output is
    that of the kernel which leaves the pooling to `pool_blocks`."""
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(d)
    T, totals = torch.bfloat16, [150, 7]
    table, k_pages = scattered_pages(rng, totals, G, d, T)
    v_pages = torch.zeros_like(k_pages)
    for s, n in enumerate(totals):
        for j in range(n):
            k_pages[table[s, j // PAGE], :, j % PAGE] = dev(rng.standard_normal((G, d)), T)
            v_pages[table[s, j // PAGE], :, j % PAGE] = dev(rng.standard_normal((G, d)), T)
    pool_table, pool_k = scattered_pages(rng, totals, G, d, T)
    pool_v, own_k, own_v = (torch.zeros_like(pool_k) for _ in range(3))
    by_kernel, by_itself = ops.Pool(pool_k, pool_v, dev(pool_table, torch.int32), size), ops.Pool(own_k, own_v, dev(pool_table, torch.int32), size)
    seq, start, dev_table = dev([0, 1], torch.int32), dev([0, 1, 2], torch.int32), dev(table, torch.int32)
    for p in range(140):
        at = [p, min(p, 6)]
        pos, q = dev(at, torch.int32), dev(rng.standard_normal((2, H * d)), T)
        outs = []
        for pool, write in ((by_itself, True), (by_kernel, False)):
            if not write:
                ops.pool_blocks(k_pages, v_pages, dev_table, pool, start, pos, 2, 1)
            scratch, out = torch.empty(2 * H * 3 * (d + 2), dtype=torch.float32, device="cuda"), torch.empty((2, H * d), dtype=T, device="cuda")
            ops.attention_capped_decode(q, k_pages, v_pages, out, scratch, seq, pos, dev_table, 2, H, G, d, d, 0.3, 0.0, None, False, 3,
                                        window=window, pool=pool, pool_write=write)
            outs.append(out)
        assert torch.equal(outs[0], outs[1]), p
        if p % 13 == 0 or p > 130:
            for a, b in ((pool_k, own_k), (pool_v, own_v)):
                assert np.allclose(f64(a), f64(b), rtol=2 ** -8, atol=1e-6), p
            n = (p + 1) // size
            assert np.allclose(read_pages(own_k, pool_table, 0, n), plain.pooled_blocks(read_pages(k_pages, table, 0, p + 1), size), rtol=2 ** -8, atol=1e-6)


@pytest.mark.parametrize("H,G,d,vd,turn,gate", [(4, 2, 16, 32, True, True), (2, 1, 128, 128, True, False), (2, 2, 64, 32, False, True), (6, 2, 32, 256, True, True)])
def test_the_split_decode_turns_its_output_back_and_gates_it(H, G, d, vd, turn, gate):
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(vd)
    T, totals = torch.bfloat16, [100, 1, 65]
    table, k_pages = scattered_pages(rng, totals, G, d, T)
    k_pages.copy_(dev(rng.standard_normal(k_pages.shape), T))
    v_pages = dev(rng.standard_normal(k_pages.shape[:-1] + (vd,)), T)
    pos, seq = dev([n - 1 for n in totals], torch.int32), dev([0, 1, 2], torch.int32)
    q, both = dev(rng.standard_normal((3, H * d)), T), dev(rng.standard_normal((3, 16 + H * vd)), T)
    a = np.arange(128)[:, None] * plain.plain_frequencies(200.0, vd)[None, :]
    cos, sin = (dev(np.cos(a), torch.float32), dev(np.sin(a), torch.float32)) if turn else (None, None)
    sinks = dev(rng.standard_normal(H), torch.float32)
    outs = []
    for fused in (True, False):
        scratch, out = torch.empty(3 * H * 2 * (vd + 2), dtype=torch.float32, device="cuda"), torch.empty((3, H * vd), dtype=T, device="cuda")
        kw = dict(back_cos=cos, back_sin=sin, gate=both[:, 16:] if gate else None) if fused else {}
        ops.attention_capped_decode(q, k_pages, v_pages, out, scratch, seq, pos, dev(table, torch.int32), 3, H, G, d, vd, 0.3, 0.0, None, True, 2,
                                    sink_values=sinks, **kw)
        outs.append(out if fused else ops.turn_back_gate(out, cos, sin, pos, both[:, 16:] if gate else None, H, vd))
    assert np.allclose(f64(outs[0]), f64(outs[1]), rtol=2e-2, atol=1e-2)


def test_pooled_blocks_that_do_not_fit_are_refused():
    import torch
    from qwen3_b200.csrc import ops
    pages = torch.zeros((2, 1, PAGE, 16), dtype=torch.float32, device="cuda")
    table = torch.zeros((1, 2), dtype=torch.int32, device="cuda")
    q, zero = torch.zeros((1, 16), dtype=torch.float32, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
    for pool, window in ((ops.Pool(pages, pages, table, 4), None), (ops.Pool(pages[:, :, :, :8], pages, table, 4), 8),
                         (ops.Pool(pages, pages, table[:, :1].contiguous(), 4), 8), (ops.Pool(pages, pages, table, 0), 8)):
        with pytest.raises(ops.KernelError, match="pooled"):
            ops.attention_generic(q, pages, pages, torch.empty_like(q), zero, zero, table, 1, 1, 1, 16, 1.0, window=window, pool=pool)


@pytest.mark.parametrize("H,G,d,vd", [(4, 2, 64, 64), (2, 1, 128, 128), (3, 3, 16, 32)])
def test_prompts_with_a_learned_sink(H, G, d, vd):
    """A number per head in the denominator - tiny for one head, towering for another - in the tiled kernels (tcgen05 where the
    head sizes allow it) and in the split decode."""
    import torch
    from qwen3_b200.csrc import ops
    rng = np.random.default_rng(d)
    T, lengths = torch.bfloat16, [300, 130, 1]
    sinks = np.array([-30.0, 12.0, 1.0, 3.5])[:H]
    sink_values = dev(sinks, torch.float32)
    table, k_pages = scattered_pages(rng, lengths, G, d, T)
    v_pages = torch.zeros(k_pages.shape[:-1] + (vd,), dtype=T, device="cuda")
    q, k, v = ([rng.standard_normal((n, h, w)) for n in lengths] for h, w in ((H, d), (G, d), (G, vd)))
    for s, n in enumerate(lengths):
        for j in range(n):
            k_pages[table[s, j // PAGE], :, j % PAGE], v_pages[table[s, j // PAGE], :, j % PAGE] = dev(k[s][j], T), dev(v[s][j], T)
    want = [plain.softmax_attention(f64(dev(q[s], T)), f64(dev(k[s], T)), f64(dev(v[s], T)), 0.3, np.tril(np.ones((n, n), dtype=bool)), sinks)
            for s, n in enumerate(lengths)]
    start, _ = packed(lengths)
    rows = dev(np.concatenate(q).reshape(-1, H * d), T)
    args = (k_pages, v_pages)
    meta = (dev(start, torch.int32), dev([0, 0, 0], torch.int32), dev(table, torch.int32), 3, max(lengths))
    outs = []
    if d == vd and d in (64, 128):
        out = torch.empty((rows.shape[0], H * vd), dtype=T, device="cuda")
        ops.attention_capped_prefill_tc(rows, *args, out, *meta, rows.shape[0], H, G, d, 0.3, 0.0, None, True, sink_values=sink_values)
        outs.append(out)
    out = torch.empty((rows.shape[0], H * vd), dtype=T, device="cuda")
    ops.attention_capped_prefill(rows, *args, out, *meta, H, G, d, vd, 0.3, 0.0, None, True, sink_values=sink_values)
    outs.append(out)
    for out in outs:
        assert np.allclose(f64(out).reshape(-1, H, vd), np.concatenate(want), atol=2e-2)
    last = dev(np.stack([q[s][-1] for s in range(3)]).reshape(3, H * d), T)
    scratch, out = torch.empty(3 * H * 2 * (vd + 2), dtype=torch.float32, device="cuda"), torch.empty((3, H * vd), dtype=T, device="cuda")
    ops.attention_capped_decode(last, *args, out, scratch, dev([0, 1, 2], torch.int32), dev([n - 1 for n in lengths], torch.int32), dev(table, torch.int32),
                                3, H, G, d, vd, 0.3, 0.0, None, True, 2, sink_values=sink_values)
    assert np.allclose(f64(out).reshape(3, H, vd), np.stack([w[-1] for w in want]), atol=2e-2)
    assert ops.tcgen05_status(torch.device("cuda")) == 0


# ============================================================================ the engine
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("vogerax")
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
        exact = plain.forward(cfg, weights, toks)
        rounded = plain.forward(cfg, weights, toks, rnd=plain.round_bf16)
        _exact[key] = (exact, 4.0 * float(np.max(np.abs(rounded - exact))) + 1e-6, float(np.abs(exact).max()))
    return _exact[key]


def check(got, requests, name, weights, dtype, label, cfg=None):
    """32-bit: every row within FP32_TOL.  bfloat16: within four times what rounding does to this very request in the plain
    implementation; a recurrent read-out followed by a unit norm is badly conditioned where the state nearly cancels, so one
    row in fifty may be further off (where the rounding falls differs from the plain run's), but none beyond four times that."""
    for rid, toks in requests.items():
        exact, bf16_tol, scale = oracle(name, weights, toks, cfg)
        tol = FP32_TOL * max(1.0, scale) if dtype == "float32" else bf16_tol
        over, rows = [], 0
        for p in range(len(toks)):
            if (rid, p) not in got:
                continue
            row = got[(rid, p)]
            rows += 1
            assert np.all(np.isfinite(row)), f"{label}: request {rid} position {p}: non-finite logits"
            err = float(np.max(np.abs(row - exact[p])))
            if dtype == "bfloat16" and tol < err <= 4.0 * tol:
                over.append(p)
                continue
            assert err <= tol, f"{label} [{dtype}] case {name}: request {rid} position {p} of {len(toks)}: {err:.3e} > {tol:.3e}"
        assert len(over) <= rows // 50, f"{label} [{dtype}] case {name}: request {rid}: {len(over)} of {rows} rows beyond {tol:.3e}: {over}"


@pytest.mark.parametrize("name", sorted(CASES))
def test_hidden_rows_after_every_layer(folders, name):
    from qwen3_b200 import StepEntry
    from qwen3_b200.parts.block import settle
    folder, weights = folders[name, "float32"]
    cfg = case(name)
    toks = random_tokens(np.random.default_rng(0), 150, cfg["vocab"])
    engine = engine_for(folder, "float32", 192, guard_scratch=True)
    seen = []

    def after_run(run, residual, pending, ctx):
        rows = residual[:ctx.n_tokens].clone()
        settle(rows, pending)
        seen.append(f64(rows))
    engine.model.after_run = after_run
    engine.step([StepEntry(engine.new_sequence(), toks, [0])])
    states = plain.hidden_states(cfg, weights, toks)
    assert len(seen) == len(states)
    for i, (got, want) in enumerate(zip(seen, states)):
        err = float(np.max(np.abs(got - want)))
        assert err <= 2e-4 * max(1.0, float(np.max(np.abs(want)))), f"case {name}: after layer {i} ({cfg['layers'][i]['type']}): {err:.3e}"
    assert engine.scratch_violations() == []


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,lengths", [("A", [1, 2, 4, 5, 6, 9, 10, 17, 18, 19, 36, 37, 38, 41, 42, 43, 64, 65, 141, 300]), ("B", [63, 64, 65, 127, 128, 129, 260]),
                                          ("C", [31, 70, 71, 72, 130, 133, 134, 150, 450]), ("D", [1, 2, 3, 4, 5, 8, 9, 10, 11, 70, 150])])
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
def test_prompt_then_token_by_token_across_windows_and_blocks(folders, name, lengths, tail, dtype):
    """The last `tail` tokens one a step, more than a window and several blocks of them: decoded tokens leave the window, become
    blocks and are seen as such, the states are carried through a long decode (a request shorter than the tail goes token
    by token from its first token)."""
    folder, weights = folders[name, dtype]
    requests = make_requests(case(name), lengths, seed=2)
    steps, rows = schedules.tail_one_by_one(requests, tail)
    engine = engine_for(folder, dtype, schedules.peak_tokens(steps))
    got = run_steps(engine, steps, rows)
    check(got, requests, name, weights, dtype, "tail one by one")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,length,cuts", [
    ("A", 260, [2, 4, 5, 7, 31, 36, 38, 41, 43, 80, 82, 120, 190, 258]), ("A", 150, list(range(2, 150, 2))),
    ("B", 230, [63, 65, 127, 129, 191, 194]), ("C", 420, [16, 69, 71, 131, 133, 203, 400]), ("D", 100, [2, 4, 6, 8, 10, 12, 50])])
def test_prompts_fed_in_portions(folders, name, length, cuts, dtype):
    """Portions of many sizes, down to two tokens, that start and end at, before and after the edges of windows, blocks and
    pages: blocks that one step begins and another finishes."""
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
    takes over their slots, pages, pooled pages and state rows.  Every row must be what the request gives alone."""
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
@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_mixed_steps_of_portions_and_single_tokens(folders, name, dtype):
    folder, weights = folders[name, dtype]
    requests = make_requests(case(name), [150, 90, 200], seed=5)
    steps, rows = schedules.mixed(requests, {"r0": 38, "r1": 41, "r2": 1}, {"r0": 1, "r1": 7, "r2": 33})
    engine = engine_for(folder, dtype, schedules.peak_tokens(steps))
    got = run_steps(engine, steps, rows)
    check(got, requests, name=name, weights=weights, dtype=dtype, label="mixed")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_long_decode_gives_pages_back_but_for_the_blocks_and_a_reused_slot_starts_from_nothing(tmp_path, dtype):
    from qwen3_b200 import StepEntry
    cfg = {"architecture": "Vogerax", "vocab": 90, "width": 48, "embedding": {"scale": 1.0}, "norm": {"eps": 1e-5, "groups": 3},
           "layers": [layer(attention(2, 1, 16, 0.3, window=50, pool=2, base=1000.0, dims=8), moe_spec(16, 3, 2, shared=8)),
                      layer(parallel(rotated(2, 1, 16, 16, 0.3, 1000.0, 8), retention(2, 8, 8, [0.9, 0.98], 100.0, 4)), None),
                      layer(attention(2, 1, 16, 0.3, window=30, pool=70, base=1000.0, dims=4, factor=2.0), dense(24))]}
    folder, weights = make_folder(tmp_path, cfg, seed=9, decided=dtype == "bfloat16")
    toks = random_tokens(np.random.default_rng(6), 330, cfg["vocab"])
    engine = engine_for(folder, dtype, 2 * 384, n_slots=1)
    for round_ in range(2):
        slot = engine.new_sequence()
        rows = [engine.step([StepEntry(slot, toks[:100], [99])])[0].cpu().numpy()]
        for p in range(100, 330):
            rows.append(engine.step([StepEntry(slot, [toks[p]], [0])])[0].cpu().numpy())
        held = [(g.need.kind, g.need.pool, g.pooled, len(g.held_pages(slot))) for g in engine.cache.groups]
        assert held == [("window", 2, False, 2), ("window", 2, True, 3), ("full", 0, False, 6), ("window", 70, False, 2), ("window", 70, True, 1)], held
        engine.release(slot)
        check({("r", 99 + i): r for i, r in enumerate(rows)}, {"r": toks}, "long decode", weights, dtype, "long decode", cfg=cfg)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["attention", "parallel", "no_pool", "no_mask", "bare_parallel"])
def test_models_of_one_kind_of_layer(tmp_path, kind, dtype):
    """Only attention with blocks (no state at all), only side-by-side layers, a window without blocks, no mask, no rotation:
    prompt, then token by token."""
    mixers = {"attention": [attention(2, 2, 16, 0.3, window=11, pool=4, base=100.0, dims=8), attention(4, 1, 32, 0.2, window=33, pool=8)],
              "parallel": [parallel(rotated(2, 1, 16, 16, 0.3, 1000.0, 8, (2.0, 32, 8.0, 1.0)), retention(2, 8, 8, [0.9, 0.7], 40.0, 8))] * 2,
              "no_pool": [attention(2, 1, 16, 0.3, window=11, base=100.0, dims=16, factor=3.0), attention(2, 2, 8, 0.3, window=70)],
              "no_mask": [attention(2, 1, 16, 0.3, base=100.0, dims=16), attention(3, 3, 8, 0.3)],
              "bare_parallel": [parallel(rotated(2, 2, 8, 12, 0.3, 50.0, 0), retention(1, 12, 8, [0.95]))]}[kind]
    cfg = {"architecture": "Vogerax", "vocab": 80, "width": 40, "embedding": {"scale": 1.5}, "norm": {"eps": 1e-5, "groups": 2},
           "layers": [layer(m, dense(48) if i % 2 else moe_spec(16, 4, 2, shared=24)) for i, m in enumerate(mixers)]}
    oracle_cfg = cfg
    if kind in ("no_pool", "no_mask"):         # the plain implementation has blocks always: blocks longer than any request are never whole
        oracle_cfg = dict(cfg, layers=[dict(l, mixer=dict(l["mixer"], mask={"size": l["mixer"].get("mask", {"size": 10 ** 6})["size"], "pool": 10 ** 6}))
                                       for l in cfg["layers"]])
    folder, weights = make_folder(tmp_path, cfg, seed=12, decided=dtype == "bfloat16")
    requests = make_requests(cfg, [90, 3], seed=13)
    steps, rows = schedules.tail_one_by_one(requests, 40)
    engine = engine_for(folder, dtype, schedules.peak_tokens(steps))
    got = run_steps(engine, steps, rows)
    check(got, requests, "one kind: " + kind, weights, dtype, "one kind", cfg=oracle_cfg)
    assert engine.cache.pages_held() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_token_is_found_again_through_its_block(tmp_path, dtype):
    """Inside a whole model: a key that stands out among hundreds.  Queries and keys read one channel of the hidden state that
    one token of the vocabulary alone sets; with that token far before the window, the last token's logits change with the
    block it lies in - and by as much as the plain implementation says."""
    import torch
    import qwen3_b200 as q
    from vogerax_cases import lively_weights
    cfg = {"architecture": "Vogerax", "vocab": 60, "width": 64, "embedding": {"scale": 1.0}, "norm": {"eps": 1e-5, "groups": 2},
           "layers": [layer(attention(2, 1, 16, 0.4, window=24, pool=4, base=1e6, dims=4), dense(48))]}
    tensors = lively_weights(q.build_model(q.config_from_dict(cfg).plan()).weight_specs(), 31)
    embed, wq, wk = tensors["embed"].float(), tensors["l0.mix.q"].float(), tensors["l0.mix.k"].float()
    embed[:, 5], embed[:, 6] = 0.0, 0.0
    embed[7, 5], embed[8, 6] = 8.0, 8.0                                  # token 7 marks its key, token 8 asks for it
    wk[10], wq[10], wq[26] = 0.0, 0.0, 0.0                               # channel 10 of a head: not rotated
    wk[10, 5], wq[10, 6], wq[26, 6] = 4.0, 4.0, 4.0
    tensors.update({"embed": embed.to(torch.bfloat16), "l0.mix.q": wq.to(torch.bfloat16), "l0.mix.k": wk.to(torch.bfloat16)})
    folder, weights = make_folder(tmp_path, cfg, seed=0, tensors=tensors)
    rng = np.random.default_rng(2)
    filler = [int(t) for t in rng.integers(9, 60, 299)]
    requests = {}
    for place in (None, 0, 3, 4, 150, 268, 271, 272, 275, 276, 290):      # the last query sees tokens from 276 and blocks 0 .. 68
        toks = list(filler)
        if place is not None:
            toks[place:place + (4 if place % 4 == 0 else 1)] = [7] * (4 if place % 4 == 0 else 1)
        requests[f"p{place}"] = toks + [8]
    logits = {}
    for schedule in (schedules.whole(requests), schedules.tail_one_by_one(requests, 33)):
        steps, rows = schedule
        engine = engine_for(folder, dtype, schedules.peak_tokens(steps))
        got = run_steps(engine, steps, rows)
        check(got, requests, "far", weights, dtype, "far", cfg=cfg)
        for rid in requests:
            logits[rid] = got[(rid, 299)]
    for place in (0, 4, 150 - 150 % 4, 268, 272, 276):
        rid = f"p{place}"
        if rid in logits:
            assert float(np.max(np.abs(logits[rid] - logits["pNone"]))) > 0.2, place      # it shows


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
            toks.append(int(np.argmax(plain.forward(cfg, weights, toks)[-1])))
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
    """bin/qwen3_chat on a Vogerax folder: the model class comes from config.json; greedy sampling through the scheduler."""
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
            toks.append(int(np.argmax(plain.forward(cfg, weights, toks)[-1])))
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
