"""Shared by the Vogerax tests: small configurations that differ in every size and option, and model folders with
weights lively enough that attention is peaked, sinks and pooled blocks carry weight and the routers decide clearly;
stored in bfloat16 so that the plain implementation reads the same values."""
import copy
import os


def attention(heads, kv_heads, dim, scale, window=None, pool=None, base=None, dims=None, factor=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if dims:
        m["rot"] = {"base": base, "dims": dims}
        if factor:
            m["rot"]["scaling"] = {"factor": factor}
    if window is not None:
        m["mask"] = {"size": window}
        if pool is not None:
            m["mask"]["pool"] = pool
    return {"type": "attention", "mixer": m}


def rotated(heads, kv_heads, dim, vdim, scale, base, dims, yarn=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dims}}
    if yarn:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return m


def retention(heads, dim, vdim, decay, base=None, dims=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}
    if dims:
        m["rot"] = {"base": base, "dims": dims}
    return m


def parallel(left, right):
    return {"type": "parallel", "mixer": {"left": left, "right": right}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, shared=None):
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        mlp["shared"] = {"ff": shared}
    return mlp


def layer(mixer, mlp, weights_of=None):
    out = dict(copy.deepcopy(mixer), mlp=copy.deepcopy(mlp))
    if weights_of is not None:
        out["weights_of"] = weights_of
    return out


# Both mixers, a window and a block that divide neither each other nor a page; values wider than keys; a layer of each kind
# that borrows another's weights (one of them from a later layer); blocks as long as their window; a layer without
# feed-forward; four parts to a norm; a shared expert of its own size.
_A0 = attention(4, 2, 16, 0.3, window=37, pool=5, base=10000.0, dims=8, factor=3.0)
_A1 = parallel(rotated(4, 2, 16, 24, 0.25, 500.0, 8, (4.0, 64, 8.0, 0.5)), retention(3, 8, 12, [0.9, 0.97, 0.5], 300.0, 8))
V_A = {
    "architecture": "Vogerax", "vocab": 211, "width": 64, "embedding": {"scale": 3.0}, "norm": {"eps": 1e-6, "groups": 4},
    "layers": [layer(_A0, moe(40, 6, 3, shared=24), weights_of=3),
               layer(_A1, dense(72)),
               layer(attention(6, 3, 8, 0.4, window=9, pool=9), None),
               layer(_A0, moe(40, 6, 3, shared=24)),
               layer(_A1, dense(72), weights_of=1)],
}
# The order the other way round; one part; one head everywhere; a window and blocks of exactly one page; blocks longer than
# their window; no shared expert; one expert; the whole head rotated; values narrower than keys; decays of 1 and 0.
V_B = {
    "architecture": "Vogerax", "vocab": 128, "width": 96, "embedding": {"scale": 0.5}, "norm": {"eps": 1e-5, "groups": 1},
    "layers": [layer(parallel(rotated(1, 1, 32, 16, 0.18, 250.0, 32), retention(1, 16, 48, [1.0])), moe(48, 1, 1)),
               layer(attention(2, 2, 16, 0.25, window=64, pool=64, base=50000.0, dims=16, factor=1.5), dense(160)),
               layer(parallel(rotated(3, 1, 16, 32, 0.3, 1000.0, 4, (2.0, 32, 4.0, 1.0)), retention(2, 32, 16, [0.0, 0.99], 10000.0, 32)), moe(32, 8, 8, shared=96)),
               layer(attention(1, 1, 32, 0.2, window=20, pool=33, base=100.0, dims=32), moe(64, 6, 2))],
}
# Sizes the tensor cores like: head sizes 64 and 128, windows of several pages, blocks of one token, more pooled blocks than
# a page holds, a state of 128 x 128.
V_C = {
    "architecture": "Vogerax", "vocab": 320, "width": 128, "embedding": {"scale": 1.0}, "norm": {"eps": 1e-5, "groups": 2},
    "layers": [layer(attention(4, 2, 64, 0.14, window=130, pool=3, base=5e5, dims=32, factor=8.0), moe(64, 8, 2, shared=64)),
               layer(parallel(rotated(4, 2, 64, 64, 0.11, 300000.0, 48, (16.0, 128, 16.0, 2.0)), retention(2, 128, 128, [0.96875, 0.999], 10000.0, 128)), dense(256)),
               layer(attention(2, 1, 128, 0.09, window=70, pool=1), moe(80, 8, 4, shared=32)),
               layer(parallel(rotated(8, 8, 128, 128, 0.09, 1e6, 128), retention(4, 16, 32, [0.5, 0.9, 0.95, 0.99], 500.0, 8)), None)],
}
# Sizes that rule out every vector path: a width that is no multiple of 4 and parts of 10 values, odd head sizes and vocabulary;
# a window of one position; two rotated values; every expert chosen.
V_D = {
    "architecture": "Vogerax", "vocab": 97, "width": 50, "embedding": {"scale": 2.0}, "norm": {"eps": 1e-5, "groups": 5},
    "layers": [layer(attention(3, 3, 6, 0.3, window=1, pool=2, base=100.0, dims=2, factor=2.0), moe(21, 4, 4, shared=11)),
               layer(parallel(rotated(2, 1, 5, 10, 0.4, 30.0, 4, (3.0, 16, 2.0, 0.7)), retention(3, 5, 9, [0.8, 0.95, 0.6], 40.0, 4)), dense(30)),
               layer(attention(4, 1, 11, 0.3, window=7, pool=3, base=1000.0, dims=10), None)],
}
CASES = {"A": V_A, "B": V_B, "C": V_C, "D": V_D}


def case(name, **changes):
    cfg = copy.deepcopy(CASES[name])
    cfg.update(changes)
    return cfg


def lively_weights(specs, seed):
    """{name: bfloat16 tensor}: matrices N(0, 1/fan_in) (routers twice that, so that choices are clear; query and key
    projections twice, so that attention is peaked), the embedding table N(0, 1), norm weights around 1, sinks
    around 1."""
    import torch
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name in sorted(specs):
        spec = specs[name]
        draw = torch.randn(spec.shape, generator=gen, dtype=torch.float32)
        tail = name.rsplit(".", 1)[-1]
        if tail == "sink":
            draw = 1.0 + 1.5 * draw
        elif spec.role == "norm":
            draw = 1.0 + 0.2 * draw
        elif tail == "router":
            draw = 2.0 * draw / (spec.shape[-1] ** 0.5)
        elif tail in ("q", "k") and ".mix." in name:
            draw = 2.0 * draw / (spec.shape[-1] ** 0.5)
        elif name != "embed":
            draw = draw / (spec.shape[-1] ** 0.5)
        out[name] = draw
    # a state that holds one token (a sequence's first) reads as (k . q) v, and the unit norm that follows keeps its sign
    # only: queries that lean towards their own keys keep k . q away from zero, where a rounding would decide
    for name in out:
        if name.endswith(".right.q"):
            out[name] = 0.8 * out[name[:-1] + "k"] + 0.6 * out[name]
    return {name: draw.to(torch.bfloat16) for name, draw in out.items()}


def decide_routers(tensors, seed):
    """Keep the routers' choices away from close calls, so that no rounded input can change them: channel 0 of the hidden
    state becomes a constant (every embedding row has it, no branch adds to it), and the routers weigh it by numbers that are
    1.5 apart, in some order, beside small weights of the other channels.  What a comparison in bfloat16 needs."""
    import torch
    gen = torch.Generator().manual_seed(seed)
    for key in list(tensors):
        t = tensors[key].float()
        if key == "embed":
            t[:, 0] = 4.0
        elif key.endswith((".norm1b", ".norm2b")):
            t[0] = 0.0
        elif key.endswith(".norm2"):
            t[0] = 1.0
        elif key.endswith(".mlp.router"):
            t = t * 0.1
            t[:, 0] = 1.5 * (torch.randperm(t.shape[0], generator=gen).float() - t.shape[0] / 2)
        tensors[key] = t.to(torch.bfloat16)
    return tensors


def make_folder(tmp_path, cfg, seed, name="model", tensors=None, decided=False):
    """Write a model folder; returns (folder, weights as float64 NumPy arrays by name)."""
    import torch
    import qwen3_b200 as q
    config = q.config_from_dict(cfg)
    if tensors is None:
        tensors = lively_weights(q.build_model(config.plan()).weight_specs(), seed)
    if decided:
        tensors = decide_routers(tensors, seed + 1)
    folder = os.path.join(str(tmp_path), name)
    q.write_model_folder(folder, config, tensors)
    return folder, {k: v.to(torch.float64).numpy() for k, v in tensors.items()}


def random_tokens(rng, n, vocab):
    return [int(t) for t in rng.integers(0, vocab, size=n)]
