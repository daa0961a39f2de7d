"""Typed configuration of the Zuretar decoder: parallel layers (one RMS norm whose output both sublayers read) listed in config.json, each
with one of two mixers and a dense or routed feed-forward or none; a layer may use another layer's weights, with a cache and state of
its own; untied output head.

  "delta"      gated delta rule: short convolutions and silu on q, k and v, unit q and k that groups of heads share, a matrix of state per
               head with one decay and one write strength per head and token
  "parallel"   two mixers side by side on the same input, half the sum of their outputs, each normed over the model's width first:
               ``left``   grouped-query softmax attention in chunks of ``mask.size`` positions, rotated (channel i paired with i + half,
                          optionally with stretched frequencies, ``rot.scaling``), q and k heads then divided by their root mean square, a
                          sink per head in the softmax denominator
               ``right``  lightning attention: a matrix of state per head with a fixed decay (``decay``), the heads normed together
  mlp "dense"  gated (silu) with biases
  mlp "moe"    routed experts without biases: sigmoid scores; ranking by score + correction inside the best-ranked blocks of experts, a block
               ranked by the sum of its two largest; weights = the picked scores as they are

config.json keys: ``architecture`` "Zuretar", ``vocab``, ``width``, ``norm.eps``, ``layers`` (per layer ``type``, ``mixer`` {sizes and
constants}, ``mlp`` {``kind`` "dense", ``ff``} or {``kind`` "moe", ``expert.ff``, ``router`` {``experts``, ``top``, ``groups`` {``count``,
``keep``}}} or null, optionally ``weights_of``: the layer whose weights it uses), optionally ``max_positions``.
Tensor names: ``embed``, ``final.norm``, ``head``, per layer with weights of its own ``l<i>.norm1``, ``l<i>.mix.*`` (``l<i>.mix.left.*`` and
``l<i>.mix.right.*`` beside each other), ``l<i>.mlp.{gate,up,down}`` with ``.b``, or ``l<i>.mlp.{e<n>.{gate,up,down}, router, correction}``.
"""
import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .base import ConfigError, LayerSpec, ModelPlan, PartSpec, optional, require

MIXERS = ("delta", "parallel")
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


def _shared_heads(m, where):
    g = optional(m, "kv_heads", int, m["heads"])
    if g <= 0 or m["heads"] % g:
        raise ConfigError(f"config.json: {where}{m['heads']} heads cannot share {g} kv_heads")


@dataclass(frozen=True)
class ZuretarConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
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
    def from_dict(cls, d, architecture="Zuretar"):
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        cfg = cls(architecture=architecture, vocab=require(d, "vocab", int), width=require(d, "width", int),
                  norm_eps=require(_section(d, "norm", ""), "eps", float), layers=copy.deepcopy(layers),
                  max_positions=optional(d, "max_positions", int, DEFAULT_MAX_POSITIONS), eos_token_id=optional(d, "eos_token_id", int, None))
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
            if layer["type"] == "delta":
                _positive(m, ("heads", "dim", "vdim", "conv"), where)
                _shared_heads(m, where)
            else:
                self._validate_pair(_section(m, "left", where), _section(m, "right", where), where)
            if layer.get("mlp") is not None:
                self._validate_mlp(layer["mlp"], where)
        for i, layer in enumerate(self.layers):
            if layer.get("weights_of") is None:
                continue
            j = self.weights_layer(i)
            mine, theirs = ({k: v for k, v in self.layers[n].items() if k != "weights_of"} for n in (i, j))
            if mine != theirs:
                raise ConfigError(f"config.json: layers[{i}] uses the weights of layers[{j}] but differs from it in more than that")

    @staticmethod
    def _validate_pair(left, right, where):
        _positive(left, ("heads", "dim", "vdim"), where + "left: ")
        _shared_heads(left, where + "left: ")
        require(left, "scale", float)
        _positive(_section(left, "mask", where + "left: "), ("size",), where + "left.mask: ")
        rot = _section(left, "rot", where + "left: ")
        dims = optional(rot, "dims", int, left["dim"])
        if dims < 0 or dims % 2 or dims > left["dim"] or not require(rot, "base", float) > 0.0:
            raise ConfigError(f"config.json: {where}left.rot: dims must be even and at most dim, base positive")
        if rot.get("scaling") is not None:
            sc = _section(rot, "scaling", where + "left.rot: ")
            if not all(require(sc, k, float) > 0.0 for k in ("factor", "original", "fast", "slow")):
                raise ConfigError(f"config.json: {where}left.rot.scaling: factor, original, fast and slow must be positive")
        _positive(right, ("heads", "dim", "vdim"), where + "right: ")
        decay = right.get("decay")
        if not isinstance(decay, list) or len(decay) != right["heads"] or any(isinstance(g, bool) or not isinstance(g, (int, float)) for g in decay):
            raise ConfigError(f"config.json: {where}right.decay must be a list of {right['heads']} numbers, one per head")

    @staticmethod
    def _validate_mlp(mlp, where):
        if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
            raise ConfigError(f"config.json: {where}mlp.kind must be 'dense' or 'moe' (or mlp null)")
        if mlp["kind"] == "dense":
            _positive(mlp, ("ff",), where + "mlp: ")
            return
        _positive(_section(mlp, "expert", where + "mlp: "), ("ff",), where + "mlp.expert: ")
        r = _section(mlp, "router", where + "mlp: ")
        _positive(r, ("experts", "top"), where + "mlp.router: ")
        if r["top"] > r["experts"]:
            raise ConfigError(f"config.json: {where}mlp.router.top exceeds the number of experts")
        if r.get("groups") is not None:
            g = _section(r, "groups", where + "mlp.router: ")
            _positive(g, ("count", "keep"), where + "mlp.router.groups: ")
            if r["experts"] % g["count"] or g["keep"] > g["count"] or r["top"] > g["keep"] * (r["experts"] // g["count"]):
                raise ConfigError(f"config.json: {where}mlp.router.groups: {r['experts']} experts do not form {g['count']} equal groups "
                                  f"of which {g['keep']} hold {r['top']} experts")

    def to_dict(self):
        d = {"architecture": self.architecture, "layers": copy.deepcopy(self.layers), "norm": {"eps": self.norm_eps}, "vocab": self.vocab,
             "width": self.width}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d

    def weights_layer(self, i):
        """The layer whose tensors layer i uses (itself, unless it says otherwise)."""
        seen = {i}
        while self.layers[i].get("weights_of") is not None:
            j = require(self.layers[i], "weights_of", int)
            if not 0 <= j < len(self.layers) or j in seen:
                raise ConfigError(f"config.json: layers[{i}]: weights_of {j} names no other layer with weights")
            seen.add(j)
            i = j
        return i

    def _mixer(self, layer):
        m, W, eps = layer["mixer"], self.width, self.norm_eps
        if layer["type"] == "delta":
            return PartSpec("gated_delta", {"hidden_size": W, "num_heads": m["heads"], "num_qk_heads": m.get("kv_heads", m["heads"]),
                                            "head_dim": m["dim"], "v_head_dim": m["vdim"], "taps": m["conv"], "eps": eps})
        left, right = m["left"], m["right"]
        rot = left["rot"]
        return PartSpec("side_by_side", {
            "hidden_size": W, "out_norms": ["mix.left.out", "mix.right.out"], "out_scale": 0.5, "eps": eps, "mixers": [
                PartSpec("masked_attention", {
                    "hidden_size": W, "num_heads": left["heads"], "num_kv_heads": left.get("kv_heads", left["heads"]), "head_dim": left["dim"],
                    "v_head_dim": left["vdim"], "scale": float(left["scale"]), "chunk": left["mask"]["size"], "qk_norm": True, "eps": eps,
                    "sink": True, "prefix": "mix.left.",
                    "position": PartSpec("rope_halves", {"head_dim": left["dim"], "rotary_dims": rot.get("dims", left["dim"]),
                                                         "theta": float(rot["base"]), "scaling": rot.get("scaling")})}),
                PartSpec("lightning", {"hidden_size": W, "num_heads": right["heads"], "head_dim": right["dim"], "v_head_dim": right["vdim"],
                                       "decay": list(right["decay"]), "eps": eps, "prefix": "mix.right."})]})

    def _feed_forward(self, mlp):
        if mlp is None:
            return PartSpec("none", {})
        if mlp["kind"] == "dense":
            return PartSpec("swiglu", {"hidden_size": self.width, "intermediate_size": mlp["ff"], "suffix": "", "bias": True,
                                       "names": {"gate": "mlp.gate", "up": "mlp.up", "down": "mlp.down"}})
        r = mlp["router"]
        groups = r.get("groups") or {}
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "intermediate_size": mlp["expert"]["ff"], "experts": r["experts"], "top": r["top"], "score": "sigmoid",
            "prefix": "mlp.", "correction": True, "groups": groups.get("count", 0), "keep": groups.get("keep", 0), "group_top": 2})

    def plan(self) -> ModelPlan:
        W = self.width

        def norm(name):
            return PartSpec("rmsnorm", {"size": W, "eps": self.norm_eps, "names": {"weight": name}})
        own = [i for i in range(len(self.layers)) if self.weights_layer(i) == i]       # the others are further runs of one of these
        layers = [LayerSpec(block="parallel_one_norm", mixer=self._mixer(self.layers[i]), feed_forward=self._feed_forward(self.layers[i].get("mlp")),
                            norms={"input": norm("norm1")}, weight_prefix=f"l{i}.") for i in own]
        return ModelPlan(
            hidden_size=W, vocab_size=self.vocab, max_positions=self.max_positions,
            embedding=PartSpec("embedding", {"vocab_size": self.vocab, "hidden_size": W, "names": {"weight": "embed"}}),
            final_norm=norm("final.norm"),
            lm_head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": W, "tied": False, "names": {"weight": "head"}}),
            layers=layers, schedule=[own.index(self.weights_layer(i)) for i in range(len(self.layers))], embedding_prefix="",
            final_norm_prefix="", lm_head_prefix="")
