"""Vinozen without a GPU: the configuration, the plan it makes, the stretches of its biases by distance, what its layers ask of
the cache, and the plain implementation against closed forms."""
import copy
import math

import numpy as np
import pytest

from plain import vinozen_plain as plain
from vinozen_cases import CASES, case, lively_weights


@pytest.mark.parametrize("name", sorted(CASES))
def test_configuration_round_trip_and_plan(name):
    import qwen3_b200 as q
    cfg = case(name)
    config = q.config_from_dict(cfg)
    assert isinstance(config, q.VinozenConfig)
    assert q.config_from_dict(config.to_dict()) == config
    plan = config.plan()
    assert [l.prefix for l in plan.layers] == [f"l{i}." for i in range(len(cfg["layers"]))] and plan.order == list(range(len(plan.layers)))
    model = q.build_model(plan)
    names, needs = set(model.weight_specs()), model.cache_needs()
    assert {"embed", "final.norm"} <= names and "head" not in names and ("side.embed" in names) == bool(cfg.get("token_side"))
    for i, layer in enumerate(cfg["layers"]):
        p, m, need, mlp = f"l{i}.", layer["mixer"], needs[i], layer["mlp"]
        assert p + "norm1" in names and (p + "norm2" in names) == (mlp is not None)
        assert ({p + "side.gate", p + "side.proj", p + "side.norm"} <= names) == bool(cfg.get("token_side"))
        if layer["type"] == "attention":
            source = m.get("kv_from")
            assert {p + "mix.q", p + "mix.o", p + "mix.rel", p + "mix.sink"} <= names
            assert ({p + "mix.k", p + "mix.v"} <= names) == (source is None) and not {p + "mix.q.norm", p + "mix.k.norm"} & names
            assert plan.layers[i].cache_from == source
            assert (need is None) if source is not None else (need.kind == "full" and need.head_dim == m["dim"] and need.state_shape == ())
        else:
            channels = m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]
            assert {p + "mix." + t for t in ("in", "conv", "conv.b", "dt_bias", "A_log", "D", "norm", "o")} <= names
            assert need.kind == "none" and need.state_shape == (m["heads"] * m["state"] * m["vdim"] + (m["conv"] - 1) * channels,)
            assert model.weight_specs()[p + "mix.in"].shape == (m["heads"] * m["vdim"] + channels + m["heads"], cfg["width"])
        if mlp is not None and mlp["kind"] == "moe":
            last = mlp["router"]["experts"] - 1
            assert {p + "mlp.router", p + "mlp.router.b", p + f"mlp.e{last}.gate", p + f"mlp.e{last}.up", p + f"mlp.e{last}.down"} <= names
            assert (p + "mlp.shared.gate" in names) == bool(mlp.get("shared")) and p + "mlp.shared.sg" not in names


@pytest.mark.parametrize("change,message", [
    (lambda c: c.pop("width"), "width"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
    (lambda c: c["embedding"].update(scale="1"), "embedding.scale"),
    (lambda c: c["token_side"].update(dim=0), "token_side.dim"),
    (lambda c: c["layers"][0].update(type="mamba"), "type"),
    (lambda c: c["layers"][0].pop("mixer"), "mixer"),
    (lambda c: c["layers"][0]["mixer"].update(groups=4), "groups"),
    (lambda c: c["layers"][0]["mixer"].update(state=300), "state"),
    (lambda c: c["layers"][0]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][0]["mixer"].update(norm_groups=7), "norm_groups"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].update(dim=300), "dim"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].pop("bias_max"), "bias_max"),
    (lambda c: c["layers"][1]["mixer"].update(bias_rows=1), "bias_rows"),
    (lambda c: c["layers"][1]["mixer"].update(bias_rows=80), "bias_rows"),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=0), "every"),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].pop("coef"), "coef"),
    (lambda c: c["layers"][5]["mixer"].update(kv_from=6), "kv_from"),
    (lambda c: c["layers"][5]["mixer"].update(kv_from=5), "kv_from"),
    (lambda c: c["layers"][5]["mixer"].update(kv_from=0), "kv_from"),
    (lambda c: c["layers"][6]["mixer"].update(kv_from=1), "heads"),
    (lambda c: c["layers"][6].update(mixer=dict(c["layers"][5]["mixer"], kv_from=5)), "no keys"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gelu"), "kind"),
    (lambda c: c["layers"][0]["mlp"].update(ff=0), "ff"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][1]["mlp"]["expert"].update(limit=0.0), "limit"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mlp"]["shared"].update(ff=0), "shared"),
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
    del bare["embedding"]
    bare["token_side"] = None
    bare["layers"][1]["mixer"]["q_temp"] = None
    bare["layers"][1]["mlp"]["shared"] = None
    bare["layers"][5]["mixer"]["kv_from"] = None
    bare["layers"][0]["mlp"] = None
    config = q.config_from_dict(bare)
    assert config.embedding_scale == 1.0 and config.side_dim is None
    model = q.build_model(config.plan())
    names = model.weight_specs()
    assert model.blocks[1].mixer.temperature is None and model.blocks[1].feed_forward.shared is None and model.blocks[1].side is None
    assert {"l5.mix.k", "l5.mix.v"} <= set(names) and "side.embed" not in names
    assert model.cache_needs()[5].kind == "full" and model.blocks[0].feed_forward is None and "l0.norm2" in model.ignorable_names()


@pytest.mark.parametrize("rows,reach", [(32, 128), (8, 16), (7, 40), (2, 3), (3, 5), (32, 17), (16, 1000), (24, 96), (12, 7.5), (64, 4096), (4, 3), (18, 72)])
def test_distances_fall_into_their_stretches(rows, reach):
    """The product's table against the plain function and, off the steps, against the formula in floating point; every distance
    exactly on a step belongs to the row it opens."""
    from fractions import Fraction
    from qwen3_b200.parts.attention import distance_buckets
    got, half = distance_buckets(rows, reach), rows // 2
    assert got[:half] == list(range(half)) and got[-1] == rows - 1 and got[-2] != rows - 1 and all(a <= b for a, b in zip(got, got[1:]))
    if reach == int(reach):
        assert got == [plain.bucket(n, rows, reach) for n in range(len(got))]
        assert all(plain.bucket(n, rows, reach) == rows - 1 for n in (len(got), 10 * len(got), 10 ** 6))
    for n in range(half, len(got) + 20):
        exact = math.log(n / half) / math.log(reach / half) * (rows - half)
        want = min(rows - 1, half + math.floor(exact))
        if abs(exact - round(exact)) > 1e-9:
            assert got[min(n, len(got) - 1)] == want, n
        else:
            k = round(exact)
            assert Fraction(n, half) ** (rows - half) >= (Fraction(reach) / half) ** k
            assert got[min(n, len(got) - 1)] == min(rows - 1, half + k), n


@pytest.mark.parametrize("rows,reach", [(1, 10), (8, 4), (8, 3), (0, 5)])
def test_tables_of_biases_that_make_no_sense_are_refused(rows, reach):
    from qwen3_b200.parts.attention import distance_buckets
    with pytest.raises(ValueError, match="biases by distance"):
        distance_buckets(rows, reach)


def test_layers_that_read_another_s_keys_share_its_pages():
    import qwen3_b200 as q
    from qwen3_b200.cache.book import CacheBook
    model = q.build_model(q.config_from_dict(case("A")).plan())
    assert model.cache_sources() == {5: 1, 6: 4}
    book = CacheBook(model.cache_needs(), 640, 320, 2)
    assert sorted(book.group_of_layer) == [1, 2, 4]              # only layers with keys of their own have pages


# ---------------------------------------------------------------- the plain implementation against closed forms
def test_state_space_is_a_sum_over_earlier_tokens():
    rng = np.random.default_rng(0)
    T, H, G, n, vd = 9, 4, 2, 3, 5
    xs, B, C = rng.standard_normal((T, H, vd)), rng.standard_normal((T, G, n)), rng.standard_normal((T, G, n))
    dt, rate, skip = rng.uniform(0.1, 2, (T, H)), rng.uniform(0.2, 3, H), rng.standard_normal(H)
    got = plain.state_space(xs, B, C, dt, rate, skip)
    for t in range(T):
        for h in range(H):
            want = skip[h] * xs[t, h]
            for s in range(t + 1):
                want = want + np.exp(-rate[h] * dt[s + 1:t + 1, h].sum()) * dt[s, h] * (B[s, h // 2] @ C[t, h // 2]) * xs[s, h]
            assert np.allclose(got[t, h], want)


def test_biased_attention_against_a_loop_over_keys():
    rng = np.random.default_rng(1)
    T, H, G, d, vd, rows, reach = 40, 4, 2, 3, 5, 6, 20
    q, k, v = rng.standard_normal((T, H, d)), rng.standard_normal((T, G, d)), rng.standard_normal((T, G, vd))
    rel, sink = rng.standard_normal((rows, H)), rng.standard_normal(H)
    got = plain.biased_attention(q, k, v, 0.7, rel, reach, sink)
    for i in (0, 1, 5, 39):
        for h in range(H):
            s = np.array([0.7 * q[i, h] @ k[j, h // 2] + rel[plain.bucket(i - j, rows, reach), h] for j in range(i + 1)])
            want = (np.exp(s)[:, None] * v[:i + 1, h // 2]).sum(0) / (np.exp(s).sum() + np.exp(sink[h]))
            assert np.allclose(got[i, h], want)


def test_convolution_sinusoid_temperature_and_norms():
    rng = np.random.default_rng(2)
    u, w, b = rng.standard_normal((7, 3)), rng.standard_normal((3, 4)), rng.standard_normal(3)
    y = plain.short_convolution(u, w, b)
    assert np.allclose(y[0], u[0] * w[:, 3] + b) and np.allclose(y[5], u[5] * w[:, 3] + u[4] * w[:, 2] + u[3] * w[:, 1] + u[2] * w[:, 0] + b)
    s = plain.sinusoid([0, 3], 5)
    assert np.allclose(s[0], [0, 1, 0, 1, 0]) and np.allclose(s[1], [math.sin(3), math.cos(3), math.sin(3 * 10000 ** -0.4), math.cos(3 * 10000 ** -0.4), math.sin(3 * 10000 ** -0.8)])
    assert np.allclose(plain.query_temperature([0, 8, 9, 19], 0.5, 10), [1.0, 1.0, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(3)])
    x = rng.standard_normal((2, 6)) + 50
    n = plain.layer_norm(x, np.ones(6), 0.0)
    assert np.allclose(n.mean(1), 0) and np.allclose((n * n).mean(1), 1)
    assert np.allclose(plain.group_rms_norm(np.array([[3.0, 3.0, 0.5, -0.5]]), np.array([1.0, 2.0, 1.0, 2.0]), 0.0, 2), [[1, 2, 1, -2]])


def test_router_and_clamped_experts():
    ids, weights = plain.route(np.array([[1.0, 3.0, 3.0, -1.0]]), 2)
    assert ids.tolist() == [[1, 2]] and np.allclose(weights, 0.5)
    w = {"gate": np.array([[5.0]]), "up": np.array([[-9.0]]), "down": np.array([[2.0]])}
    assert np.allclose(plain.clamped(np.array([[1.0]]), w, "", 1.5), 2.0 * 1.5 * plain.sigmoid(1.702 * 1.5) * (-1.5 + 1.0))
    w["gate"][:] = -5.0                                       # a gate is bounded from above only
    assert np.allclose(plain.clamped(np.array([[1.0]]), w, "", 1.5), 2.0 * -5.0 * plain.sigmoid(-1.702 * 5.0) * (-0.5))


@pytest.mark.parametrize("name", sorted(CASES))
def test_the_plain_model_is_causal(name):
    import torch
    import qwen3_b200 as q
    cfg = case(name)
    specs = q.build_model(q.config_from_dict(cfg).plan()).weight_specs()
    w = {k: v.to(torch.float64).numpy() for k, v in lively_weights(specs, 5).items()}
    toks = [int(t) for t in np.random.default_rng(3).integers(0, cfg["vocab"], 12)]
    a, b = plain.logits(toks, w, cfg), plain.logits(toks[:7] + [(t + 1) % cfg["vocab"] for t in toks[7:]], w, cfg)
    assert np.all(np.isfinite(a)) and np.allclose(a[:7], b[:7]) and not np.allclose(a[7:], b[7:])
    assert copy.deepcopy(a).std() > 0.1
