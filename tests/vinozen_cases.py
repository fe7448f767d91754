"""Shared by the Vinozen tests: small configurations that differ in every size and option, and model folders with weights
lively enough that attention is peaked, sinks and biases by distance carry weight, states decay at different speeds and the
routers decide clearly; stored in bfloat16 so that the plain implementation reads the same values."""
import copy
import os


def attention(heads, kv_heads, dim, vdim, scale, bias_max, temp=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def mamba2(heads, vdim, state, groups, conv, norm_groups):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, limit, experts, top, shared=None):
    mlp = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        mlp["shared"] = {"ff": shared[0], "limit": shared[1]}
    return mlp


def layer(mixer, mlp):
    return dict(copy.deepcopy(mixer), mlp=copy.deepcopy(mlp))


# Both mixers, two sources of keys with readers of other scales and temperatures, values wider than keys, a layer without
# feed-forward, sizes off the tensor cores' steps beside sizes on them.
V_A = {
    "architecture": "Vinozen", "vocab": 211, "width": 64, "embedding": {"scale": 3.0}, "norm": {"eps": 1e-6}, "token_side": {"dim": 16},
    "layers": [layer(mamba2(6, 12, 20, 3, 4, 2), dense(72)),
               layer(attention(4, 2, 16, 32, 0.9, 40, temp=(0.5, 7)), moe(40, 1.5, 6, 3, shared=(24, 0.7))),
               layer(attention(4, 2, 16, 32, 0.6, 100), None),
               layer(mamba2(4, 16, 16, 1, 2, 1), moe(32, 2.0, 5, 2)),
               layer(attention(6, 3, 16, 16, 1.1, 9, temp=(1.0, 64), kv_from=None), dense(40)),
               layer(attention(4, 2, 16, 32, 1.2, 17, temp=(0.2, 3), kv_from=1), moe(40, 1.5, 6, 3, shared=(24, 0.7))),
               layer(attention(6, 3, 16, 16, 0.8, 300, kv_from=4), dense(24))],
}
# Attention first, one head everywhere, a group per head, a convolution of one tap, a norm part per head, one expert, no side
# input, no scale of the embedding, biases that reach five tokens.
V_B = {
    "architecture": "Vinozen", "vocab": 128, "width": 96, "norm": {"eps": 1e-5},
    "layers": [layer(attention(1, 1, 32, 16, 0.7, 5), moe(48, 1.0, 1, 1)),
               layer(mamba2(3, 32, 48, 3, 1, 3), moe(32, 3.0, 8, 8, shared=(96, 2.0))),
               layer(attention(1, 1, 32, 16, 0.4, 64, temp=(0.7, 1), kv_from=0), dense(160)),
               layer(mamba2(1, 64, 16, 1, 3, 1), None)],
}
# Sizes the tensor cores like: head sizes 64 and 128, states of 128 x 64 and 32 x 48.
V_C = {
    "architecture": "Vinozen", "vocab": 320, "width": 128, "embedding": {"scale": 1.0}, "norm": {"eps": 1e-5}, "token_side": {"dim": 32},
    "layers": [layer(attention(4, 2, 64, 64, 0.5, 128, temp=(0.3, 100)), moe(64, 2.0, 8, 2, shared=(64, 1.0))),
               layer(mamba2(4, 64, 128, 2, 4, 4), dense(256)),
               layer(attention(2, 1, 128, 128, 0.3, 90), moe(96, 1.2, 8, 4, shared=(32, 3.0))),
               layer(mamba2(6, 48, 32, 1, 4, 2), moe(64, 2.0, 4, 1)),
               layer(attention(2, 1, 128, 128, 0.4, 200, temp=(0.4, 50), kv_from=2), None)],
}
# Sizes that rule out every vector path: an odd width and vocabulary, odd head sizes, a convolution of five taps.
V_D = {
    "architecture": "Vinozen", "vocab": 97, "width": 51, "embedding": {"scale": 2.0}, "norm": {"eps": 1e-5}, "token_side": {"dim": 5},
    "layers": [layer(mamba2(3, 7, 5, 1, 5, 3), moe(21, 1.0, 4, 4, shared=(11, 2.5))),
               layer(attention(3, 3, 5, 10, 0.8, 12, temp=(0.9, 10)), dense(30)),
               layer(attention(4, 1, 11, 3, 0.6, 30), None),
               layer(attention(3, 3, 5, 10, 0.5, 7.5, kv_from=1), moe(20, 2.0, 3, 2))],
}
CASES = {"A": V_A, "B": V_B, "C": V_C, "D": V_D}
BIAS_ROWS = (8, 16, 7, 10, 16, 24, 32)       # the rows of a layer's table of biases, by the layer's number


def case(name, **changes):
    cfg = copy.deepcopy(CASES[name])
    cfg.update(changes)
    return cfg


def lively_weights(specs, seed):
    """{name: bfloat16 tensor}: matrices N(0, 1/fan_in) (those that read the hidden state less, it is not normed before a
    layer), the embedding table N(0, 1), norm weights around 1, sinks around 1, biases by distance N(0, 1.5), steps from slow to
    fast."""
    import torch
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name in sorted(specs):
        spec = specs[name]
        tail = name.rsplit(".", 1)[-1]
        shape = spec.shape
        if tail == "rel":
            shape = (BIAS_ROWS[int(name.split(".")[0][1:]) % len(BIAS_ROWS)], shape[1])
        draw = torch.randn(shape, generator=gen, dtype=torch.float32)
        if tail in ("sink", "D"):
            draw = 1.0 + 1.5 * draw
        elif tail == "rel":
            draw = 1.5 * draw
        elif tail == "dt_bias":
            draw = draw - 2.0
        elif tail == "A_log":
            draw = draw * 0.8 + 0.5
        elif name.endswith(("conv.b", "router.b")):
            draw = 0.5 * draw
        elif tail == "conv":
            draw = draw / spec.shape[-1] ** 0.5
        elif spec.role == "norm":
            draw = 1.0 + 0.2 * draw
        elif name not in ("embed", "side.embed"):
            draw = draw / (spec.shape[-1] ** 0.5)
            if tail in ("in", "gate", "up", "v", "router"):
                draw = 0.4 * draw
        out[name] = draw.to(torch.bfloat16)
    return out


def decide_routers(tensors, seed):
    """Keep the routers' choices away from close calls, so that no rounded input can change them: the last channel of the hidden
    state becomes nearly constant (every embedding row has it, its sinusoid hardly turns, no branch adds to it), and the
    routers weigh it by numbers that are 1.5 apart, in some order, beside small weights of the other channels.  What a
    comparison in bfloat16 needs."""
    import torch
    gen = torch.Generator().manual_seed(seed)
    for key in list(tensors):
        t = tensors[key].float()
        if key == "embed":
            t[:, -1] = 4.0
        elif key.endswith((".norm1", ".norm2", ".side.norm")):
            t[-1] = 0.0
        elif key.endswith(".mlp.router"):
            t = t * 0.1
            t[:, -1] = 1.5 * (torch.randperm(t.shape[0], generator=gen).float() - t.shape[0] / 2)
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
