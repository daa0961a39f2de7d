"""Typed configuration of the Ramupel decoder: parallel layers (one layer norm without bias whose output both sublayers read) listed
in config.json; every sublayer's result passes a gate per channel before it joins the stream, and what goes on from a layer is a
weighted sum over the depth, of the embedding output and everything the layers have left so far; the head is the embedding table.

  "latent_attention"  causal softmax attention whose keys and values are made per head from one cached latent per token beside one
                      rotated key part that all heads share (channel i paired with i + half); queries straight from the input; a
                      sigmoid gate per head on the heads' outputs
  "gla"               gated linear attention: a matrix of state per head, a decay per key channel from a low-rank projection
  mlp "dense"         ungated, with the activation xIELU and its two learned numbers

config.json keys: ``architecture`` "Ramupel", ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``layers`` (per layer ``type``,
``mixer`` {sizes and constants}, ``mlp`` {``kind`` "dense", ``ff``} or null), optionally ``max_positions``.
Tensor names: ``embed``, ``final.norm``, per layer ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.{up,down,act}``, ``l<i>.rg1``, ``l<i>.rg1.b``,
``l<i>.rg2``, ``l<i>.rg2.b``, ``l<i>.dwa``.
"""
import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .base import ConfigError, LayerSpec, ModelPlan, PartSpec, optional, require

MIXERS = ("latent_attention", "gla")
DEFAULT_MAX_POSITIONS = 1 << 17


def _section(d, key, where):
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}'{key}' must be an object")
    return v


def _positive(m, keys, where):
    for k in keys:
        if require(m, k, int) <= 0:
            raise ConfigError(f"config.json: {where}'{k}' must be positive")


@dataclass(frozen=True)
class RamupelConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float = 1.0
    layers: List[Dict[str, Any]] = field(default_factory=list)
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_id: Optional[int] = None

    # what the command line and the benchmark ask any configuration
    @property
    def vocab_size(self):
        return self.vocab

    @property
    def hidden_size(self):
        return self.width

    @property
    def num_hidden_layers(self):
        return len(self.layers)

    @classmethod
    def from_dict(cls, d, architecture="Ramupel"):
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        emb = {} if d.get("embedding") is None else _section(d, "embedding", "")
        cfg = cls(architecture=architecture, vocab=require(d, "vocab", int), width=require(d, "width", int),
                  norm_eps=require(_section(d, "norm", ""), "eps", float), embedding_scale=optional(emb, "scale", float, 1.0),
                  layers=copy.deepcopy(layers), max_positions=optional(d, "max_positions", int, DEFAULT_MAX_POSITIONS),
                  eos_token_id=optional(d, "eos_token_id", int, None))
        cfg.validate()
        return cfg

    def validate(self):
        if self.vocab <= 0 or self.width <= 0 or self.max_positions <= 0 or not self.norm_eps > 0.0:
            raise ConfigError("config.json: vocab, width, max_positions and norm.eps must be positive")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]: "
            if not isinstance(layer, dict) or layer.get("type") not in MIXERS:
                raise ConfigError(f"config.json: {where}'type' must be one of {MIXERS}")
            m = _section(layer, "mixer", where)
            _positive(m, ("heads", "dim", "vdim"), where)
            if layer["type"] == "latent_attention":
                _positive(m, ("kv_rank", "rot_dim"), where)
                require(m, "scale", float)
                rot = _section(m, "rot", where)
                if m["rot_dim"] % 2 or optional(rot, "dims", int, m["rot_dim"]) != m["rot_dim"] or not require(rot, "base", float) > 0.0:
                    raise ConfigError(f"config.json: {where}rot_dim must be even, rot.dims equal to it, rot.base positive")
            elif not require(m, "tau", float) > 0.0:
                raise ConfigError(f"config.json: {where}tau must be positive")
            mlp = layer.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
                    raise ConfigError(f"config.json: {where}mlp.kind must be 'dense' (or mlp null)")
                _positive(mlp, ("ff",), where + "mlp: ")

    def to_dict(self):
        d = {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale}, "layers": copy.deepcopy(self.layers),
             "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d

    def _mixer(self, layer):
        m, W, eps = layer["mixer"], self.width, self.norm_eps
        if layer["type"] == "gla":
            return PartSpec("gated_linear", {"hidden_size": W, "num_heads": m["heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"],
                                             "tau": float(m["tau"]), "eps": eps})
        return PartSpec("latent_attention", {
            "hidden_size": W, "num_heads": m["heads"], "head_dim": m["dim"], "rot_dim": m["rot_dim"], "v_head_dim": m["vdim"],
            "kv_rank": m["kv_rank"], "q_rank": None, "scale": float(m["scale"]), "eps": eps, "out_gate": "head",
            "position": PartSpec("rope_halves", {"head_dim": m["rot_dim"], "rotary_dims": m["rot_dim"], "theta": float(m["rot"]["base"])})})

    def _feed_forward(self, mlp):
        if mlp is None:
            return PartSpec("none", {})
        return PartSpec("dense", {"hidden_size": self.width, "intermediate_size": mlp["ff"], "activation": "xielu"})

    def plan(self) -> ModelPlan:
        W = self.width

        def norm(name):
            return PartSpec("layernorm", {"size": W, "eps": self.norm_eps, "names": {"weight": name}, "has_bias": False})
        layers = [LayerSpec(block="parallel_depth", mixer=self._mixer(layer), feed_forward=self._feed_forward(layer.get("mlp")),
                            norms={"input": norm("norm1")}, weight_prefix=f"l{i}.", block_params={"depth": i + 2})
                  for i, layer in enumerate(self.layers)]
        return ModelPlan(
            hidden_size=W, vocab_size=self.vocab, max_positions=self.max_positions,
            embedding=PartSpec("embedding", {"vocab_size": self.vocab, "hidden_size": W, "names": {"weight": "embed"}, "scale": self.embedding_scale}),
            final_norm=norm("final.norm"),
            lm_head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": W, "tied": True, "names": {"weight": "head"}}),
            layers=layers, schedule=list(range(len(layers))), embedding_prefix="", final_norm_prefix="", lm_head_prefix="", depth_average=True)
