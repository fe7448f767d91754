"""Typed configuration of the Vogerax decoder, read from its config.json.

A Vogerax model is a list of layers on a float32 hidden state with a norm before and after every sublayer,
x += norm1b(mixer(norm1(x))) and then x += norm2b(ff(norm2(x))); the norms are RMS norms over equal parts of the row.
What the file gives, key by key:

  architecture        "Vogerax"
  vocab, width        sizes of the embedding table and of the hidden state
  embedding.scale     the embedding's rows are multiplied by it
  norm.eps, .groups   eps of every norm (inside the root); the parts that a layer's norms and the final norm split a row into
  layers[i].type      "attention": mixer {heads, kv_heads, dim, vdim, scale, rot {base, dims, scaling {factor}}, mask {size, pool}}:
                      grouped-query attention whose values are its projected keys, with linearly scaled rotation and a
                      sliding window of `size` tokens beside which every block of `pool` earlier tokens is seen as one mean
                      "parallel": mixer {left {...}, right {...}}: half the sum of two mixers that read the same input, each
                      output normed first; left {heads, kv_heads, dim, vdim, scale, rot {base, dims, scaling {factor,
                      original, fast, slow}}}: attention over every earlier key with normed queries and keys, YaRN,
                      rotated values, a learned sink and an output gate; right {heads, dim, vdim, decay [heads],
                      rot {base, dims}}: retention with a fixed decay per head
  layers[i].mlp       {kind "dense", ff} | {kind "moe", expert {ff}, router {experts, top}, shared {ff}} | null; every
                      feed-forward is W_down max(W_up x, 0)^2
  layers[i].weights_of   j: the layer has no tensors of its own and runs with layer j's, on a cache and state of its own

Optional keys (`mlp`, `mask`, `rot`, `rot.scaling`, `shared`, `weights_of`) may be null or absent: the mechanism is then not
there.  The file has no bound on positions and no stop tokens.  `plan()` states the model as data for the parts, the
cache and the step function.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Optional

from .dozazen import MAX_POSITIONS, _get, _opt
from .plan import LayerSpec, ModelPlan, PartSpec
from .registry import ConfigError, register_architecture

MAX_ROUTER = 1023              # what the router kernel takes


@dataclass(frozen=True)
class VogeraxConfig:
    vocab: int
    width: int
    embedding_scale: float
    norm_eps: float
    norm_groups: int
    layers: List[Dict[str, Any]]            # as in the file, checked
    torch_dtype: str = "bfloat16"

    architecture = "Vogerax"

    @classmethod
    def from_dict(cls, root: dict) -> "VogeraxConfig":
        if not isinstance(root, dict):
            raise ConfigError("model config root must be a JSON object")
        name = root.get("architecture", (root.get("architectures") or [None])[0])
        if name != cls.architecture:
            raise ConfigError(f"only {cls.architecture} is read by this class, not {name!r}")
        layers = root.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config field 'layers' must be a non-empty array")
        embedding = _opt(root, "embedding", dict) or {}
        norm = _get(root, "norm", dict)
        groups = _opt(norm, "groups", int, "norm.")
        scale = _opt(embedding, "scale", float, "embedding.")
        config = cls(
            vocab=_get(root, "vocab", int),
            width=_get(root, "width", int),
            embedding_scale=1.0 if scale is None else scale,
            norm_eps=_get(norm, "eps", float, "norm."),
            norm_groups=1 if groups is None else groups,
            layers=copy.deepcopy(layers),
            torch_dtype=_opt(root, "torch_dtype", str) or "bfloat16",
        )
        config.validate()
        return config

    # -- checks
    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0:
            raise ConfigError("vocab and width must be positive")
        if not self.norm_eps > 0:
            raise ConfigError("norm.eps must be positive")
        if self.norm_groups <= 0 or self.width % self.norm_groups:
            raise ConfigError("norm.groups must divide width")
        if self.torch_dtype not in ("bfloat16", "float32"):
            raise ConfigError("torch_dtype is bfloat16 or float32")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]."
            if not isinstance(layer, dict):
                raise ConfigError(f"{where[:-1]} must be an object")
            kind = _get(layer, "type", str, where)
            m, w = _get(layer, "mixer", dict, where), where + "mixer."
            if kind == "attention":
                self._check_attention(m, w)
                if m["vdim"] != m["dim"]:
                    raise ConfigError(f"{w}vdim: the values are the keys, of their size")
                mask = _opt(m, "mask", dict, w)
                if mask is not None and (_get(mask, "size", int, w + "mask.") <= 0 or (_opt(mask, "pool", int, w + "mask.") or 0) < 0):
                    raise ConfigError(f"{w}mask: size must be positive and pool must not be negative")
            elif kind == "parallel":
                left, right = _get(m, "left", dict, w), _get(m, "right", dict, w)
                self._check_attention(left, w + "left.")
                if left["vdim"] % 2:
                    raise ConfigError(f"{w}left.vdim must be even (rotated values)")
                if not isinstance(left.get("rot"), dict):
                    raise ConfigError(f"{w}left.rot must be an object: the values turn by its base")
                self._check_retention(right, w + "right.")
            else:
                raise ConfigError(f"{where}type: 'attention' or 'parallel', not {kind!r}")
            mlp = _opt(layer, "mlp", dict, where)
            if mlp is not None:
                self._check_mlp(mlp, where + "mlp.")
            owner = self.owner_of(i)
            if owner != i and layer["type"] != self.layers[owner].get("type"):
                raise ConfigError(f"{where}weights_of: layer {owner} is of another type")

    def owner_of(self, i: int) -> int:
        """The layer whose tensors layer i runs with."""
        seen = set()
        while True:
            where = f"layers[{i}]."
            if i in seen:
                raise ConfigError(f"{where}weights_of goes round in a circle")
            seen.add(i)
            owner = _opt(self.layers[i], "weights_of", int, where)
            if owner is None:
                return i
            if not 0 <= owner < len(self.layers) or not isinstance(self.layers[owner], dict):
                raise ConfigError(f"{where}weights_of must name another layer")
            i = owner

    @staticmethod
    def _check_rot(m: dict, w: str) -> None:
        rot = _opt(m, "rot", dict, w)
        if rot is None:
            return
        dims = _get(rot, "dims", int, w + "rot.")
        if dims < 0 or dims % 2 or dims > m["dim"]:
            raise ConfigError(f"{w}rot.dims must be even and at most dim")
        if _get(rot, "base", float, w + "rot.") <= 0:
            raise ConfigError(f"{w}rot.base must be positive")
        scaling = _opt(rot, "scaling", dict, w + "rot.")
        if scaling is not None:
            for key in VogeraxConfig._scaling_keys(scaling):
                if not _get(scaling, key, float, w + "rot.scaling.") > 0:
                    raise ConfigError(f"{w}rot.scaling.{key} must be positive")

    @staticmethod
    def _scaling_keys(scaling: dict):
        """A ramp over the pairs (YaRN) has `original`, `fast` and `slow`; without them every frequency is divided alike."""
        return ("factor", "original", "fast", "slow") if "original" in scaling else ("factor",)

    @staticmethod
    def _check_attention(m: dict, w: str) -> None:
        heads, kv = _get(m, "heads", int, w), _get(m, "kv_heads", int, w)
        dim, vdim = _get(m, "dim", int, w), _get(m, "vdim", int, w)
        if heads <= 0 or kv <= 0 or heads % kv or not 0 < dim <= 256 or not 0 < vdim <= 256:
            raise ConfigError(f"{w}heads must be a multiple of kv_heads, dim and vdim up to 256")
        if not _get(m, "scale", float, w) > 0:
            raise ConfigError(f"{w}scale must be positive")
        VogeraxConfig._check_rot(m, w)

    @staticmethod
    def _check_retention(m: dict, w: str) -> None:
        heads, dim, vdim = _get(m, "heads", int, w), _get(m, "dim", int, w), _get(m, "vdim", int, w)
        if heads <= 0 or not 0 < dim <= 256 or not 0 < vdim <= 256:
            raise ConfigError(f"{w}heads must be positive, dim and vdim up to 256")
        decay = m.get("decay")
        if not isinstance(decay, list) or len(decay) != heads or any(isinstance(v, bool) or not isinstance(v, (int, float)) for v in decay):
            raise ConfigError(f"{w}decay must hold one number per head")
        if any(not 0 <= v <= 1 for v in decay):
            raise ConfigError(f"{w}decay: numbers from 0 to 1")
        VogeraxConfig._check_rot(m, w)

    @staticmethod
    def _check_mlp(mlp: dict, where: str) -> None:
        kind = _get(mlp, "kind", str, where)
        if kind == "dense":
            if _get(mlp, "ff", int, where) <= 0:
                raise ConfigError(f"{where}ff must be positive")
            return
        if kind != "moe":
            raise ConfigError(f"{where}kind: 'dense' or 'moe', not {kind!r}")
        if _get(_get(mlp, "expert", dict, where), "ff", int, where + "expert.") <= 0:
            raise ConfigError(f"{where}expert.ff must be positive")
        shared = _opt(mlp, "shared", dict, where)
        if shared is not None and _get(shared, "ff", int, where + "shared.") <= 0:
            raise ConfigError(f"{where}shared.ff must be positive")
        r, w = _get(mlp, "router", dict, where), where + "router."
        experts, top = _get(r, "experts", int, w), _get(r, "top", int, w)
        if not 0 < top <= experts or experts > MAX_ROUTER:
            raise ConfigError(f"{w}needs 0 < top <= experts <= {MAX_ROUTER}")

    def to_dict(self) -> dict:
        """The keys of a config.json that `from_dict` reads back to an equal object."""
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.norm_eps, "groups": self.norm_groups},
                "layers": copy.deepcopy(self.layers), "torch_dtype": self.torch_dtype}

    # -- the model as data
    @staticmethod
    def _position(rot: Optional[dict], head_dim: int) -> Optional[PartSpec]:
        if not rot or not rot.get("dims"):
            return None
        scaling = rot.get("scaling")
        if scaling:
            keys = VogeraxConfig._scaling_keys(scaling)
            scaling = dict({k: float(scaling[k]) for k in keys}, kind="yarn" if len(keys) > 1 else "linear")
        return PartSpec("rope", {"head_dim": head_dim, "theta": float(rot["base"]), "max_positions": MAX_POSITIONS,
                                 "rotary_dim": rot["dims"], "scaling": scaling or None, "theta_float32": False})

    def _pooled_attention(self, m: dict) -> PartSpec:
        mask = m.get("mask") or {}
        return PartSpec("gqa_attention", {
            "hidden_size": self.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
            "scale": float(m["scale"]), "position": self._position(m.get("rot"), m["dim"]), "window": mask.get("size"),
            "pool": mask.get("pool") or 0, "tied_values": True, "prefix": "mix.", "names": {"q": "q", "k": "k", "o": "o"}})

    def _rotated_value_attention(self, m: dict) -> PartSpec:
        return PartSpec("gqa_attention", {
            "hidden_size": self.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
            "value_dim": m["vdim"], "scale": float(m["scale"]), "position": self._position(m.get("rot"), m["dim"]),
            "qk_norm": PartSpec("rms_norm", {"size": m["dim"], "eps": self.norm_eps}), "norm_once": True,
            "value_position": self._position({"base": m["rot"]["base"], "dims": m["vdim"]}, m["vdim"]),
            "learned_sink": True, "out_gate": True, "prefix": "mix.left.",
            "names": {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "out_gate": "g", "sink": "sink"}})

    def plan(self) -> ModelPlan:
        H, eps = self.width, self.norm_eps
        norm = PartSpec("rms_norm", {"size": H, "eps": eps, "groups": self.norm_groups})
        owners = [i for i in range(len(self.layers)) if self.owner_of(i) == i]
        layers = []
        for i in owners:
            layer = self.layers[i]
            m, mlp = layer["mixer"], layer.get("mlp")
            if layer["type"] == "attention":
                mixer = self._pooled_attention(m)
            else:
                r = m["right"]
                retention = PartSpec("retention", {
                    "hidden_size": H, "num_heads": r["heads"], "head_dim": r["dim"], "value_dim": r["vdim"],
                    "decay": [float(v) for v in r["decay"]], "eps": eps, "position": self._position(r.get("rot"), r["dim"]),
                    "k_scale": r["dim"] ** -0.5, "prefix": "mix.right."})
                mixer = PartSpec("parallel_mixers", {
                    "hidden_size": H, "mixers": [self._rotated_value_attention(m["left"]), retention], "scales": [0.5, 0.5],
                    "out_norms": ["mix.left.out", "mix.right.out"], "eps": eps})
            feed_forward = None
            if mlp is not None and mlp["kind"] == "dense":
                feed_forward = PartSpec("dense_mlp", {"hidden_size": H, "intermediate_size": mlp["ff"], "prefix": "mlp.",
                                                      "activation": "relu2", "names": {"up": "up", "down": "down"}})
            elif mlp is not None:
                r = mlp["router"]
                feed_forward = PartSpec("routed_experts", {
                    "hidden_size": H, "intermediate_size": mlp["expert"]["ff"], "experts": r["experts"], "top": r["top"],
                    "expert_activation": "relu2", "shared_size": (mlp.get("shared") or {}).get("ff"), "shared_gate": False,
                    "correction": False, "prefix": "mlp."})
            layers.append(LayerSpec(block=PartSpec("sandwich_norm", {"norm": norm}), mixer=mixer, feed_forward=feed_forward,
                                    prefix=f"l{i}."))
        order, caches, extra = [], [], len(layers)
        for i in range(len(self.layers)):
            order.append(owners.index(self.owner_of(i)))
            if self.owner_of(i) == i:
                caches.append(order[-1])
            else:                                            # borrowed weights, a cache or state of its own
                caches.append(extra)
                extra += 1
        return ModelPlan(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=H, max_positions=MAX_POSITIONS,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": H, "scale": self.embedding_scale,
                                                   "tensor": ""}),
            embedding_prefix="embed", layers=layers, order=order, caches=caches, residual_dtype="float32",
            final_norm=norm, final_norm_prefix="final.", final_norm_name="final.norm",
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": H, "tensor": ""}),
            head_prefix="head", stop_token_ids=[],
        )


register_architecture(VogeraxConfig.architecture, VogeraxConfig)
