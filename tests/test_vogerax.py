"""Vogerax without a GPU: the configuration, the plan it makes, the frequencies of its rotations, the cache's bookkeeping
for pooled blocks, and the plain implementation against closed forms."""
import copy
import math

import numpy as np
import pytest

from plain import vogerax_plain as plain
from vogerax_cases import CASES, case, decide_routers, lively_weights

PAGE = 64


@pytest.mark.parametrize("name", sorted(CASES))
def test_configuration_round_trip_and_plan(name):
    import qwen3_b200 as q
    cfg = case(name)
    config = q.config_from_dict(cfg)
    assert isinstance(config, q.VogeraxConfig)
    assert q.config_from_dict(config.to_dict()) == config
    plan = config.plan()
    owners = [i for i, l in enumerate(cfg["layers"]) if l.get("weights_of") is None]
    assert [l.prefix for l in plan.layers] == [f"l{i}." for i in owners] and len(plan.order) == len(cfg["layers"])
    assert plan.order == [owners.index(l.get("weights_of", i)) for i, l in enumerate(cfg["layers"])]
    assert len(set(plan.caches)) == len(cfg["layers"])                    # every run has a cache or state of its own
    model = q.build_model(plan)
    names, needs = set(model.weight_specs()), model.cache_needs()
    assert {"embed", "final.norm", "head"} <= names
    for i, layer in enumerate(cfg["layers"]):
        p, m, need = f"l{layer.get('weights_of', i)}.", layer["mixer"], needs[plan.cache_of_run(i)]
        assert (f"l{i}.norm1" in names) == (i in owners)
        assert {p + "norm1", p + "norm1b"} <= names and (p + "norm2b" in names) == (layer["mlp"] is not None)
        if layer["type"] == "attention":
            mask = m["mask"]
            assert {p + "mix.q", p + "mix.k", p + "mix.o"} <= names and p + "mix.v" not in names
            assert need.kind == "window" and need.window == max(mask["size"], mask["pool"]) and need.pool == mask["pool"]
            assert need.state_shape == ()
        else:
            right = m["right"]
            assert {p + "mix.left." + t for t in ("q", "k", "v", "o", "g", "sink", "q.norm", "k.norm", "out")} <= names
            assert {p + "mix.right." + t for t in ("q", "k", "v", "o", "g", "out")} <= names
            assert need.kind == "full" and need.pool == 0 and need.state_shape == (right["heads"] * right["dim"] * right["vdim"],)
        mlp = layer["mlp"]
        if mlp is not None and mlp["kind"] == "moe":
            last = mlp["router"]["experts"] - 1
            assert {p + "mlp.router", p + f"mlp.e{last}.up", p + f"mlp.e{last}.down"} <= names
            assert (p + "mlp.shared.up" in names) == bool(mlp.get("shared"))
            assert not {p + "mlp.correction", p + "mlp.e0.gate", p + "mlp.shared.gate", p + "mlp.shared.sg"} & names
        elif mlp is not None:
            assert {p + "mlp.up", p + "mlp.down"} <= names and p + "mlp.gate" not in names


@pytest.mark.parametrize("change,message", [
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
    (lambda c: c["norm"].update(groups=3), "groups"),
    (lambda c: c["norm"].update(groups=0), "groups"),
    (lambda c: c["embedding"].update(scale="1"), "embedding.scale"),
    (lambda c: c["layers"][1].update(type="hgrn2"), "type"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=16), "vdim"),
    (lambda c: c["layers"][2]["mixer"].update(dim=300, vdim=300), "dim"),
    (lambda c: c["layers"][2]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(size=0), "mask"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(pool=-1), "pool"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(base=0.0), "rot.base"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0.0), "factor"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(vdim=25), "vdim"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(rot=None), "rot"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.5, 0.5]), "decay"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.5, 0.5, 1.5]), "decay"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][1]["mlp"].update(kind="gelu"), "kind"),
    (lambda c: c["layers"][1]["mlp"].update(ff=0), "ff"),
    (lambda c: c["layers"][3]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][3]["mlp"]["shared"].update(ff=0), "shared"),
    (lambda c: c["layers"][0].update(weights_of=9), "weights_of"),
    (lambda c: c["layers"][0].update(weights_of=1), "weights_of"),
    (lambda c: c["layers"][3].update(weights_of=0), "circle"),
])
def test_configuration_faults_are_named(change, message):
    import qwen3_b200 as q
    cfg = case("A")
    change(cfg)
    with pytest.raises(q.ConfigError, match=message):
        q.config_from_dict(cfg)


def test_optional_mechanisms_may_be_absent_or_null():
    import qwen3_b200 as q
    bare = case("A")
    del bare["embedding"], bare["norm"]["groups"]
    bare["layers"][1]["mixer"]["left"]["rot"].update(scaling=None, dims=0)
    bare["layers"][1]["mixer"]["right"]["rot"] = None
    bare["layers"][2]["mixer"]["mask"] = None
    bare["layers"][3]["mixer"]["mask"].pop("pool")
    bare["layers"][3]["mixer"]["rot"] = None
    bare["layers"][3]["mlp"]["shared"] = None
    for i in (0, 4):
        bare["layers"][i] = copy.deepcopy(bare["layers"][{0: 3, 4: 1}[i]])
        bare["layers"][i]["weights_of"] = None
    config = q.config_from_dict(bare)
    assert config.embedding_scale == 1.0 and config.norm_groups == 1
    model = q.build_model(config.plan())
    needs = model.cache_needs()
    assert needs[2].kind == "full" and needs[3].kind == "window" and needs[3].pool == 0 and needs[3].window == 37
    left, right = model.blocks[1].mixer.mixers
    assert left.position is None and left.value_position is not None and right.position is None and model.blocks[3].mixer.position is None
    assert "l3.mlp.shared.up" not in model.weight_specs() and "l4.mix.left.q" in model.weight_specs()


def test_a_layer_may_borrow_from_one_that_borrows():
    import qwen3_b200 as q
    cfg = case("A")
    cfg["layers"].append(dict(copy.deepcopy(cfg["layers"][0]), weights_of=0))
    plan = q.config_from_dict(cfg).plan()
    assert plan.order[5] == plan.order[3] == plan.order[0] and len(set(plan.caches)) == 6


@pytest.mark.parametrize("dims,base,scaling", [(8, 500.0, (4.0, 64, 8.0, 0.5)), (64, 1e6, (32.0, 4096, 32.0, 1.0)), (4, 30.0, (3.0, 16, 2.0, 0.7)),
                                               (128, 10000.0, (2.0, 2048, 64.0, 0.25)), (2, 100.0, (5.0, 8, 3.0, 2.9)), (16, 70.0, (8.0, 10, 900.0, 0.001))])
def test_frequencies_of_scaled_rotations(dims, base, scaling):
    """The product's tables against the plain functions; the ramp reaches both ends, and beyond them frequencies are whole
    or divided."""
    import torch
    from qwen3_b200.parts.position import RotaryEmbedding
    yarn = dict(zip(("factor", "original", "fast", "slow"), scaling))
    part = RotaryEmbedding(dims + 3, base, 1 << 20, rotary_dim=dims, scaling=dict(yarn, kind="yarn"), theta_float32=False)
    freq, magnitude = plain.yarn(base, dims, yarn)
    assert np.allclose(part.frequencies(), freq, rtol=1e-12) and math.isclose(part.magnitude(), magnitude)
    own = plain.plain_frequencies(base, dims)
    assert np.all(freq <= own * (1 + 1e-12)) and np.all(freq >= own / yarn["factor"] * (1 - 1e-12))
    part.prepare(300, torch.device("cpu"))
    angle = np.arange(300)[:, None] * freq[None, :]
    assert np.allclose(part.cos.double().numpy(), magnitude * np.cos(angle), atol=3e-7)
    assert np.allclose(part.sin.double().numpy(), magnitude * np.sin(angle), atol=3e-7)
    linear = RotaryEmbedding(dims, base, 1 << 20, scaling={"kind": "linear", "factor": 4.0}, theta_float32=False)
    assert np.allclose(linear.frequencies(), own / 4.0, rtol=1e-12) and linear.magnitude() == 1.0
    with pytest.raises(ValueError, match="kind"):
        RotaryEmbedding(dims, base, 10, scaling={"kind": "none", "factor": 2.0})


# ---------------------------------------------------------------- the cache's bookkeeping
def test_the_book_keeps_pages_of_pooled_blocks_for_good():
    from qwen3_b200.cache import CacheBook, CacheNeed
    needs = [CacheNeed("window", 1, 8, window=45, pool=5), CacheNeed("window", 1, 8, window=45), CacheNeed("window", 1, 8, window=70, pool=70),
             CacheNeed("window", 1, 8, window=45, pool=5), CacheNeed("window", 2, 8, window=45, pool=1)]
    book = CacheBook(needs, max_tokens=12 * PAGE, max_seq_len=12 * PAGE, n_slots=2)
    assert [g.pooled for g in book.groups] == [False, True, False, False, True, False, True]
    assert book.group_of_layer == {0: 0, 1: 2, 2: 3, 3: 0, 4: 5} and book.pool_group_of_layer == {0: 1, 2: 4, 3: 1, 4: 6}
    assert [g.n_pages for g in book.groups] == [12, 12 // 5 + 2, 12, 12, 2, 12, 12]      # a pool of blocks is as large as it can need to be
    slot = book.alloc_slot()

    def step(n):
        book.reserve([(slot, n)])
        book.commit([(slot, n)])

    def held():
        return [sorted(int(i) for i in np.nonzero(g.table[slot] >= 0)[0]) for g in book.groups]
    step(4)
    assert [len(h) for h in held()] == [1, 0, 1, 1, 0, 1, 1]               # no whole block of five yet
    step(1)
    assert len(held()[1]) == 1
    step(5 * PAGE)                                                          # 325 tokens: 65 blocks of five, 4 of seventy, 325 of one
    assert held() == [[4, 5], [0, 1], [4, 5], [4, 5], [0], [4, 5], [0, 1, 2, 3, 4, 5]]
    for _ in range(PAGE):
        step(1)
    assert held()[0] == [5, 6] and held()[1] == [0, 1] and held()[6] == list(range(7))
    before = held()
    book.reserve([(slot, 3 * PAGE)])
    book.cancel([(slot, 3 * PAGE)])                                         # the step did not run: its pages go back, of blocks too
    assert held() == before
    book.free_slot(slot)
    assert all(g.n_free == g.n_pages for g in book.groups)


@pytest.mark.parametrize("window,pool", [(1, 2), (7, 3), (37, 5), (64, 64), (20, 33), (130, 3), (5, 200)])
def test_the_tokens_of_an_unfinished_block_stay(window, pool):
    """Whatever the steps' sizes, the pages that hold a token that a later step reads - inside a later query's window, or in a
    block that is not finished yet - are there."""
    from qwen3_b200.cache import CacheBook
    from qwen3_b200.parts.attention import GQAAttention
    part = GQAAttention(16, 1, 1, 8, 1.0, window=window, pool=pool, tied_values=True)
    book = CacheBook([part.cache_need()], max_tokens=40 * PAGE, max_seq_len=40 * PAGE, n_slots=1)
    slot, rng, length = book.alloc_slot(), np.random.default_rng(window), 0
    while length < 1500:
        n = int(rng.integers(1, 90))
        book.reserve([(slot, n)])
        table = book.groups[0].table[slot]
        first_query = length
        first_block = length // pool                                       # blocks from here on are made by this step
        for p in list(range(max(0, first_query - window + 1), length + n)) + list(range(first_block * pool, length)):
            assert table[p // PAGE] >= 0, (length, p)
        pool_row = book.groups[1].table[slot]
        for b in range((length + n) // pool):
            assert pool_row[b // PAGE] >= 0
        book.commit([(slot, n)])
        length += n


def test_pools_never_run_out_before_the_tokens_do():
    """Any mix of sequences whose tokens fit fits with its blocks: the pool's size is a bound."""
    from qwen3_b200.cache import CacheBook, CacheFull, CacheNeed
    rng = np.random.default_rng(3)
    for pool in (1, 2, 7, 64, 100):
        for slots in (1, 3, 9):
            book = CacheBook([CacheNeed("full", 1, 8), CacheNeed("window", 1, 8, window=max(8, pool), pool=pool)], max_tokens=20 * PAGE,
                             max_seq_len=20 * PAGE, n_slots=slots)
            held = [book.alloc_slot() for _ in range(slots)]
            while True:
                slot, n = held[int(rng.integers(slots))], int(rng.integers(1, 2 * PAGE))
                try:
                    book.reserve([(slot, n)])
                except CacheFull:
                    need = -(-(book.length(slot) + n) // PAGE) - -(-book.length(slot) // PAGE)
                    assert need > book.groups[0].n_free or book.length(slot) + n > book.max_seq_len
                    break
                book.commit([(slot, n)])


def test_pooled_blocks_need_a_window_that_covers_one():
    from qwen3_b200.cache import CacheNeed
    from qwen3_b200.parts.attention import GQAAttention
    for bad in (dict(kind="full", pool=4), dict(kind="window", window=3, pool=4)):
        with pytest.raises(ValueError, match="pooled"):
            CacheNeed(num_kv_heads=1, head_dim=8, **bad)
    with pytest.raises(ValueError, match="pooled"):
        GQAAttention(16, 1, 1, 8, 1.0, pool=4)
    with pytest.raises(ValueError, match="keys"):
        GQAAttention(16, 1, 1, 8, 1.0, value_dim=16, tied_values=True)


# ---------------------------------------------------------------- the plain implementation against closed forms
def test_visibility_of_tokens_and_blocks():
    tokens, blocks = plain.visible(30, 5, 3)
    for i in range(30):
        seen = [j for j in range(30) if tokens[i, j]]
        assert seen == list(range(max(0, i - 4), i + 1))
        whole = [b for b in range(10) if all(3 * b + t <= i - 5 for t in range(3))]
        assert [b for b in range(10) if blocks[i, b]] == whole
    assert blocks.sum() > 0 and plain.visible(4, 2, 9)[1].shape == (4, 0)


def test_blocks_of_equal_tokens_weigh_as_one():
    """All keys and values of a block alike: its mean is any of them, and it enters the softmax once."""
    T, P, window = 9, 4, 3
    k = np.zeros((T, 1, 2))
    v = np.arange(T, dtype=float)[:, None, None] * np.ones((1, 1, 1))
    v[:4] = 7.0
    tokens, blocks = plain.visible(T, window, P)
    keys, values = np.concatenate([k, plain.pooled_blocks(k, P)]), np.concatenate([v, plain.pooled_blocks(v, P)])
    out = plain.softmax_attention(np.zeros((T, 1, 2)), keys, values, 1.0, np.concatenate([tokens, blocks], axis=1))
    assert np.isclose(out[5, 0, 0], (7 + 4 + 5) / 3)              # 3, 4 and 5 in the window; the first block not seen yet
    assert np.isclose(out[6, 0, 0], (4 + 5 + 6 + 7) / 4)          # the first block, 0 .. 3, has left the window
    assert np.isclose(out[8, 0, 0], (6 + 7 + 8 + 7) / 4)          # 4 and 5 are seen neither as tokens nor as a block


def test_a_sink_takes_its_share_and_scores_shift_out():
    rng = np.random.default_rng(0)
    q, k, v = (rng.standard_normal((5, 2, 3)) for _ in range(3))
    causal = np.tril(np.ones((5, 5), dtype=bool))
    none = plain.softmax_attention(q, k, v, 0.7, causal)
    sink = np.array([-1e9, 2.0])
    got = plain.softmax_attention(q, k, v, 0.7, causal, sink)
    assert np.allclose(got[:, 0], none[:, 0])
    for i in range(5):
        s = np.exp((k[:i + 1, 1] @ q[i, 1]) * 0.7)
        assert np.allclose(got[i, 1], none[i, 1] * s.sum() / (s.sum() + math.exp(2.0)))


def test_rotated_values_depend_on_distances_only():
    """One key: the output is the value turned by the distance; position by itself does not show."""
    rng = np.random.default_rng(1)
    v = rng.standard_normal((1, 1, 6))
    freq = plain.plain_frequencies(50.0, 6)
    for j, i in ((0, 4), (100, 104)):
        out = plain.rotary(plain.rotary(v, [j], freq), [i], freq, sign=-1.0)
        assert np.allclose(out, plain.rotary(v, [4], freq, sign=-1.0))
    assert np.allclose(plain.rotary(v, [9], freq, magnitude=1.5), 1.5 * plain.rotary(v, [9], freq))


def test_retention_equals_its_sum_form():
    rng = np.random.default_rng(2)
    T, H, d, vd, width = 20, 2, 6, 4, 10
    m = {"heads": H, "dim": d, "vdim": vd, "decay": [0.9, 0.4], "rot": {"base": 60.0, "dims": 4}}
    w = {n: rng.standard_normal((H * s, width)) for n, s in (("q", d), ("k", d), ("v", vd), ("g", vd))}
    w["o"] = np.eye(H * vd)
    h = rng.standard_normal((T, width))
    got = plain.retention(h, w, "", m, 1e-6)
    freq = plain.plain_frequencies(60.0, 4)
    q, k = (plain.rotary((h @ w[n].T).reshape(T, H, d), range(T), freq) for n in ("q", "k"))
    v = (h @ w["v"].T).reshape(T, H, vd)
    o = np.zeros((T, H, vd))
    for a in range(H):
        for t in range(T):
            for j in range(t + 1):
                o[t, a] += m["decay"][a] ** (t - j) * (q[t, a] @ k[j, a]) / math.sqrt(d) * v[j, a]
    want = plain.rms_unit(o, 1e-6).reshape(T, H * vd) * plain.silu(h @ w["g"].T)
    assert np.allclose(got, want, rtol=1e-8, atol=1e-8)


def test_norm_in_groups_is_a_norm_of_every_part():
    x = np.array([[3.0, 4.0, 0.0, 0.5]])
    got = plain.group_norm(x, np.array([1.0, 2.0, 1.0, 1.0]), 0.0, 2)
    assert np.allclose(got, [[3 / math.sqrt(12.5), 8 / math.sqrt(12.5), 0.0, 0.5 / math.sqrt(0.125)]])
    assert np.allclose(plain.group_norm(x, np.ones(4), 1e-3, 1), plain.rms_norm(x, np.ones(4), 1e-3))


def test_router_weighs_by_plain_scores_of_all_experts():
    w = {"router": np.eye(4)}
    h = np.array([[2.0, 0.0, 1.0, -3.0]])
    ids, weights = plain.route(h, w, "", {"experts": 4, "top": 2})
    s = np.exp(h[0]) / np.exp(h[0]).sum()
    assert list(ids[0]) == [0, 2] and np.allclose(weights[0], s[[0, 2]]) and weights.sum() < 1.0


def test_decided_routers_are_far_from_close_calls():
    import qwen3_b200 as q
    for name in sorted(CASES):
        cfg = case(name)
        tensors = decide_routers(lively_weights(q.build_model(q.config_from_dict(cfg).plan()).weight_specs(), 5), 6)
        w = {k: v.double().numpy() for k, v in tensors.items()}
        toks = [int(t) for t in np.random.default_rng(4).integers(0, cfg["vocab"], 150)]
        margins, route = [], plain.route

        def watched(h, w, p, r, rnd=plain.same):
            z = np.sort(h @ w[p + "router"].T, axis=1)
            if r["top"] < r["experts"]:
                margins.append(float(np.min(z[:, -r["top"]] - z[:, -r["top"] - 1])))
            return route(h, w, p, r, rnd)
        plain.route = watched
        try:
            plain.forward(cfg, w, toks)
        finally:
            plain.route = route
        assert all(m > 0.1 for m in margins), (name, margins)


def test_the_plain_model_is_causal():
    import qwen3_b200 as q
    cfg = case("A")
    tensors = lively_weights(q.build_model(q.config_from_dict(cfg).plan()).weight_specs(), 7)
    w = {k: v.double().numpy() for k, v in tensors.items()}
    toks = [int(t) for t in np.random.default_rng(5).integers(0, cfg["vocab"], 90)]
    full = plain.forward(cfg, w, toks)
    assert np.allclose(plain.forward(cfg, w, toks[:53]), full[:53], rtol=1e-9, atol=1e-9)
    assert copy.deepcopy(cfg) == case("A")
