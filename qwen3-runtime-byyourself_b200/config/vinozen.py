"""Typed configuration of the Vinozen decoder, read from its config.json.

A Vinozen model is a list of layers on a float32 hidden state with a layer norm (a weight, no bias) on every sublayer's output,
x += norm1(mixer(x)) and then x += norm2(ff(x)); after them every layer adds a gated slice of a second embedding of the
token.  Positions enter as sinusoids beside the token's embedding and as biases by distance in the attention; nothing is
rotated.  The output projection is the embedding table.  What the file gives, key by key:

  architecture        "Vinozen"
  vocab, width        sizes of the embedding table and of the hidden state
  embedding.scale     the embedding's rows are multiplied by it (the sinusoids are not)
  norm.eps            eps of every norm (inside the root)
  token_side.dim      width of a layer's slice of the second embedding `side.embed` [vocab, layers * dim]
  layers[i].type      "attention": mixer {heads, kv_heads, dim, vdim, scale, bias_max, q_temp {coef, every}, kv_from}:
                      grouped-query attention over every earlier key with queries and keys at unit rms per head, a query
                      temperature that grows with the position, a learned bias by distance (far distances in stretches that
                      grow by equal factors up to bias_max; the rows of the table are the tensor's, `bias_rows` states
                      them where no checkpoint does) and a learned sink;
                      kv_from j: the layer has no keys and values of its own and reads layer j's
                      "mamba2": mixer {heads, vdim, state, groups, conv, norm_groups}: a selective state space with a short
                      convolution of `conv` taps and a gate before a norm in groups
  layers[i].mlp       {kind "dense", ff}: W_down (SiLU(W_gate x) * W_up x)
                      | {kind "moe", expert {ff, limit}, router {experts, top}, shared {ff, limit}}: clamped experts chosen by
                      biased logits, and a shared one | null

Optional keys (`embedding`, `token_side`, `mlp`, `mlp.shared`, `q_temp`, `kv_from`, `bias_rows`) may be null or absent: the mechanism is then
not there.  The file has no bound on positions and no stop tokens.  `plan()` states the model as data for the parts, the
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
SHARED_SIZES = ("heads", "kv_heads", "dim", "vdim")     # what a layer has in common with the one whose keys it reads


@dataclass(frozen=True)
class VinozenConfig:
    vocab: int
    width: int
    embedding_scale: float
    norm_eps: float
    side_dim: Optional[int]
    layers: List[Dict[str, Any]]            # as in the file, checked
    torch_dtype: str = "bfloat16"

    architecture = "Vinozen"

    @classmethod
    def from_dict(cls, root: dict) -> "VinozenConfig":
        if not isinstance(root, dict):
            raise ConfigError("model config root must be a JSON object")
        name = root.get("architecture", (root.get("architectures") or [None])[0])
        if name != cls.architecture:
            raise ConfigError(f"only {cls.architecture} is read by this class, not {name!r}")
        layers = root.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config field 'layers' must be a non-empty array")
        embedding = _opt(root, "embedding", dict) or {}
        scale = _opt(embedding, "scale", float, "embedding.")
        side = _opt(root, "token_side", dict)
        config = cls(
            vocab=_get(root, "vocab", int),
            width=_get(root, "width", int),
            embedding_scale=1.0 if scale is None else scale,
            norm_eps=_get(_get(root, "norm", dict), "eps", float, "norm."),
            side_dim=_get(side, "dim", int, "token_side.") if side is not None else None,
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
        if self.torch_dtype not in ("bfloat16", "float32"):
            raise ConfigError("torch_dtype is bfloat16 or float32")
        if self.side_dim is not None and self.side_dim <= 0:
            raise ConfigError("token_side.dim must be positive")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]."
            if not isinstance(layer, dict):
                raise ConfigError(f"{where[:-1]} must be an object")
            kind = _get(layer, "type", str, where)
            m, w = _get(layer, "mixer", dict, where), where + "mixer."
            if kind == "attention":
                self._check_attention(m, w)
                self._check_source(i, m, w)
            elif kind == "mamba2":
                self._check_state_space(m, w)
            else:
                raise ConfigError(f"{where}type: 'attention' or 'mamba2', not {kind!r}")
            mlp = _opt(layer, "mlp", dict, where)
            if mlp is not None:
                self._check_mlp(mlp, where + "mlp.")

    @staticmethod
    def _check_attention(m: dict, w: str) -> None:
        heads, kv = _get(m, "heads", int, w), _get(m, "kv_heads", int, w)
        dim, vdim = _get(m, "dim", int, w), _get(m, "vdim", int, w)
        if heads <= 0 or kv <= 0 or heads % kv or not 0 < dim <= 256 or not 0 < vdim <= 256:
            raise ConfigError(f"{w}heads must be a multiple of kv_heads, dim and vdim up to 256")
        if not _get(m, "scale", float, w) > 0:
            raise ConfigError(f"{w}scale must be positive")
        if not _get(m, "bias_max", float, w) > 0:
            raise ConfigError(f"{w}bias_max must be positive")
        rows = _opt(m, "bias_rows", int, w)
        if rows is not None and (rows < 2 or m["bias_max"] <= rows // 2):
            raise ConfigError(f"{w}bias_rows: at least two, and half of them below bias_max")
        temp = _opt(m, "q_temp", dict, w)
        if temp is not None:
            _get(temp, "coef", float, w + "q_temp.")
            if _get(temp, "every", int, w + "q_temp.") <= 0:
                raise ConfigError(f"{w}q_temp.every must be positive")

    def _check_source(self, i: int, m: dict, w: str) -> None:
        source = _opt(m, "kv_from", int, w)
        if source is None:
            return
        other = self.layers[source] if 0 <= source < i else None
        if not isinstance(other, dict) or other.get("type") != "attention":
            raise ConfigError(f"{w}kv_from must name an earlier attention layer")
        if other["mixer"].get("kv_from") is not None:
            raise ConfigError(f"{w}kv_from: layer {source} has no keys and values of its own")
        if any(other["mixer"][k] != m[k] for k in SHARED_SIZES):
            raise ConfigError(f"{w}kv_from: the heads of layer {source} are others")

    @staticmethod
    def _check_state_space(m: dict, w: str) -> None:
        heads, vdim, state, groups = (_get(m, k, int, w) for k in ("heads", "vdim", "state", "groups"))
        if heads <= 0 or groups <= 0 or heads % groups or not 0 < vdim <= 256 or not 0 < state <= 256:
            raise ConfigError(f"{w}heads must be a multiple of groups, vdim and state up to 256")
        if not 0 < _get(m, "conv", int, w) <= 64:
            raise ConfigError(f"{w}conv: 1 to 64 taps")
        parts = _get(m, "norm_groups", int, w)
        if parts <= 0 or heads * vdim % parts:
            raise ConfigError(f"{w}norm_groups must divide heads * vdim")

    @staticmethod
    def _check_clamped(expert: dict, w: str) -> None:
        if _get(expert, "ff", int, w) <= 0 or not _get(expert, "limit", float, w) > 0:
            raise ConfigError(f"{w}ff and limit must be positive")

    @staticmethod
    def _check_mlp(mlp: dict, where: str) -> None:
        kind = _get(mlp, "kind", str, where)
        if kind == "dense":
            if _get(mlp, "ff", int, where) <= 0:
                raise ConfigError(f"{where}ff must be positive")
            return
        if kind != "moe":
            raise ConfigError(f"{where}kind: 'dense' or 'moe', not {kind!r}")
        VinozenConfig._check_clamped(_get(mlp, "expert", dict, where), where + "expert.")
        shared = _opt(mlp, "shared", dict, where)
        if shared is not None:
            VinozenConfig._check_clamped(shared, where + "shared.")
        r, w = _get(mlp, "router", dict, where), where + "router."
        experts, top = _get(r, "experts", int, w), _get(r, "top", int, w)
        if not 0 < top <= experts or experts > MAX_ROUTER:
            raise ConfigError(f"{w}needs 0 < top <= experts <= {MAX_ROUTER}")

    def to_dict(self) -> dict:
        """The keys of a config.json that `from_dict` reads back to an equal object."""
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.norm_eps},
                "token_side": {"dim": self.side_dim} if self.side_dim is not None else None,
                "layers": copy.deepcopy(self.layers), "torch_dtype": self.torch_dtype}

    # -- the model as data
    def _attention(self, m: dict) -> PartSpec:
        return PartSpec("gqa_attention", {
            "hidden_size": self.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
            "value_dim": m["vdim"], "scale": float(m["scale"]), "norm_once": True,
            "qk_norm": PartSpec("rms_norm", {"size": m["dim"], "eps": self.norm_eps, "weighted": False}),
            "temperature": dict(m["q_temp"]) if m.get("q_temp") else None, "distance_bias": m["bias_max"],
            "bias_rows": m.get("bias_rows"), "learned_sink": True, "shared_kv": m.get("kv_from") is not None, "prefix": "mix.",
            "names": {"q": "q", "k": "k", "v": "v", "o": "o", "rel": "rel", "sink": "sink"}})

    def _state_space(self, m: dict) -> PartSpec:
        return PartSpec("state_space", {
            "hidden_size": self.width, "num_heads": m["heads"], "value_dim": m["vdim"], "state": m["state"], "groups": m["groups"],
            "taps": m["conv"], "norm_groups": m["norm_groups"], "eps": self.norm_eps, "prefix": "mix."})

    def _feed_forward(self, mlp: Optional[dict]) -> Optional[PartSpec]:
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return PartSpec("swiglu", {"hidden_size": self.width, "intermediate_size": mlp["ff"], "prefix": "mlp.",
                                       "names": {"gate": "gate", "up": "up", "down": "down"}})
        shared = mlp.get("shared") or {}
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "intermediate_size": mlp["expert"]["ff"], "experts": mlp["router"]["experts"],
            "top": mlp["router"]["top"], "limit": float(mlp["expert"]["limit"]), "scoring": "top_logits", "router_bias": True,
            "shared_size": shared.get("ff"), "shared_limit": shared.get("limit"), "shared_gate": False, "prefix": "mlp."})

    def plan(self) -> ModelPlan:
        H, n = self.width, len(self.layers)
        norm = PartSpec("layer_norm", {"size": H, "eps": self.norm_eps})
        layers = []
        for i, layer in enumerate(self.layers):
            m, side = layer["mixer"], None
            if self.side_dim is not None:
                side = {"table": "side.embed", "vocab": self.vocab, "columns": n * self.side_dim, "dim": self.side_dim,
                        "index": i, "eps": self.norm_eps, "gate": "side.gate", "proj": "side.proj", "norm": "side.norm"}
            layers.append(LayerSpec(
                block=PartSpec("post_norm", {"norm": norm, "hidden_size": H, "side": side}),
                mixer=self._attention(m) if layer["type"] == "attention" else self._state_space(m),
                feed_forward=self._feed_forward(layer.get("mlp")), prefix=f"l{i}.",
                cache_from=m.get("kv_from") if layer["type"] == "attention" else None))
        return ModelPlan(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=H, max_positions=MAX_POSITIONS,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": H, "scale": self.embedding_scale,
                                                   "tensor": "", "positions": "sinusoid"}),
            embedding_prefix="embed", layers=layers, order=list(range(n)), residual_dtype="float32",
            final_norm=norm, final_norm_prefix="final.", final_norm_name="final.norm",
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": H, "tied_to": "embed", "tensor": ""}),
            head_prefix="head", stop_token_ids=[],
        )


register_architecture(VinozenConfig.architecture, VinozenConfig)
