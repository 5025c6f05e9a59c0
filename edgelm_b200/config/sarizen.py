"""The Sarizen decoder's configuration, from its own config.json keys.

config.json: `architecture` "Sarizen", `vocab`, `width`, `norm.eps`, `logit_scale` (absent: 1) and `layers`, one entry per layer:
`type` ("lightning" or "latent_attention"), `mixer` (its sizes and constants) and `mlp` (a dense or a mixture-of-experts
feed-forward, or null for none).  Optional: `max_positions`.  Tensors: `embed`, `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.*`, `l<i>.mlp.*`,
`final.norm`, `head`.

A layer is x += mixer(norm1(x)) + mlp(norm2(x)), both sublayers reading the same x (block "parallel_prenorm").
  lightning          linear attention with a constant decay per head (`parts/lightning.py`): `heads`, `dim`, `vdim`, `decay` (one a head)
  latent_attention   softmax attention over a shared low-rank latent (`parts/latent_attention.py`): `heads`, `dim` unrotated and `rot_dim`
                     rotated dimensions a query head, `vdim`, `kv_rank`, `scale`, `rot` {dims, base, scaling {factor, original, fast, slow}}
                     (neighbouring pairs, the wavelengths stretched by YaRN; no scaling: none), `mask` {size} (a sliding window;
                     absent: causal), a sink in the softmax and a sigmoid gate per head on the output
The feed-forward: {"kind": "dense", "ff"}: squared ReLU without a gate (`parts/squared_relu.py`);
{"kind": "moe", "expert": {ff}, "router": {experts, top}, "shared": {ff}}: gated experts, scored by a sigmoid each, whose scores, as they
are, multiply the experts' inputs; a shared expert is added as it is (`parts/moe.py`).
"""
from dataclasses import dataclass
from typing import Any, Mapping, Tuple

from .base import ConfigError, LayerSpec, ModelPlan, PartSpec, ScheduleEntry, optional, require
from .registry import register_architecture

DEFAULT_MAX_POSITIONS = 1 << 20


def _sub(d, key, where, needed=True):
    v = d.get(key)
    if v is None and not needed:
        return None
    if not isinstance(v, Mapping):
        raise ConfigError(f"{where}: key '{key}' should be an object, found {v!r}")
    return v


@register_architecture("Sarizen", model_type="sarizen")
@dataclass(frozen=True)
class SarizenConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[Mapping[str, Any], ...]
    logit_scale: float = 1.0
    max_positions: int = DEFAULT_MAX_POSITIONS

    architecture = "Sarizen"

    @classmethod
    def from_dict(cls, d):
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' should be a non-empty list")
        cfg = cls(vocab=require(d, "vocab", int), width=require(d, "width", int),
                  eps=require(_sub(d, "norm", "config.json"), "eps", float, "config.json norm"), layers=tuple(layers),
                  logit_scale=optional(d, "logit_scale", float, 1.0), max_positions=optional(d, "max_positions", int, DEFAULT_MAX_POSITIONS))
        if cfg.vocab <= 0 or cfg.width <= 0 or cfg.max_positions <= 0 or not cfg.eps > 0:
            raise ConfigError("config.json: vocab, width, max_positions and norm.eps must be positive")
        cfg.plan()     # every layer's keys are read and checked here
        return cfg

    def to_dict(self):
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
               "layers": [dict(l) for l in self.layers]}
        if self.logit_scale != 1.0:
            out["logit_scale"] = self.logit_scale
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        return out

    # ------------------------------------------------------------------ mixers
    def _lightning(self, m, where):
        heads = require(m, "heads", int, where)
        decay = m.get("decay")
        if not isinstance(decay, (list, tuple)) or len(decay) != heads or not all(isinstance(a, (int, float)) and not isinstance(a, bool) for a in decay):
            raise ConfigError(f"{where}: key 'decay' should list one number per head ({heads})")
        dim = require(m, "dim", int, where)
        return PartSpec("decay_linear_attention", {
            "hidden_size": self.width, "heads": heads, "head_dim": dim, "v_head_dim": optional(m, "vdim", int, None, where) or dim,
            "decay": tuple(float(a) for a in decay), "activation": "silu", "eps": self.eps,
            "names": {"q": "mix.q", "k": "mix.k", "v": "mix.v", "g": "mix.g", "norm": "mix.norm", "o": "mix.o"}})

    def _latent(self, m, where):
        dim, rot_dim = require(m, "dim", int, where), require(m, "rot_dim", int, where)
        rot, mask = _sub(m, "rot", where), _sub(m, "mask", where, needed=False)
        scaling = _sub(rot, "scaling", where + " rot", needed=False)
        if require(rot, "dims", int, where + " rot") != rot_dim:
            raise ConfigError(f"{where} rot: {rot['dims']} dimensions, but rot_dim is {rot_dim}")
        return PartSpec("latent_attention", {
            "hidden_size": self.width, "num_heads": require(m, "heads", int, where), "head_dim": dim, "rot_dim": rot_dim,
            "v_head_dim": optional(m, "vdim", int, None, where) or dim, "kv_rank": require(m, "kv_rank", int, where),
            "scale": require(m, "scale", float, where), "eps": self.eps, "rot_base": require(rot, "base", float, where + " rot"),
            "rot_scaling": {k: require(scaling, k, float, where + " rot scaling") for k in ("factor", "original", "fast", "slow")}
                           if scaling is not None else None,
            "rot_pairs": "interleaved", "head_gate": True,
            "mask": {"kind": "window", "size": require(mask, "size", int, where + " mask")} if mask is not None else None,
            "names": {"q": "mix.q", "dkv": "mix.dkv", "dkv_norm": "mix.dkv.norm", "uk": "mix.uk", "uv": "mix.uv", "o": "mix.o",
                      "gate": "mix.g", "sink": "mix.sink"}})

    # ------------------------------------------------------------------ feed-forwards
    def _mlp(self, mlp, where):
        kind = require(mlp, "kind", str, where)
        if kind == "dense":
            return PartSpec("squared_relu", {"hidden_size": self.width, "intermediate_size": require(mlp, "ff", int, where),
                                             "names": {"up": "mlp.up", "down": "mlp.down"}})
        if kind != "moe":
            raise ConfigError(f"{where}: kind '{kind}' is not part of this architecture (dense, moe)")
        e, r, shared = _sub(mlp, "expert", where), _sub(mlp, "router", where), _sub(mlp, "shared", where, needed=False)
        return PartSpec("moe", {
            "hidden_size": self.width, "intermediate_size": require(e, "ff", int, where + " expert"),
            "experts": require(r, "experts", int, where + " router"), "top": require(r, "top", int, where + " router"),
            "router": {"kind": "scored", "score": "sigmoid", "renormalize": False}, "weight_on": "input",
            "shared": PartSpec("swiglu", {"hidden_size": self.width, "intermediate_size": require(shared, "ff", int, where + " shared"),
                                          "names": {"gate": "mlp.shared.gate", "up": "mlp.shared.up", "down": "mlp.shared.down"}})
                      if shared is not None else None,
            "names": {"expert": "mlp.e", "gate": "gate", "up": "up", "down": "down", "router": "mlp.router"}})

    def _layer(self, i, layer):
        where = f"config.json layers[{i}]"
        if not isinstance(layer, Mapping):
            raise ConfigError(f"{where} should be an object")
        kind = require(layer, "type", str, where)
        mixers = {"lightning": self._lightning, "latent_attention": self._latent}
        if kind not in mixers:
            raise ConfigError(f"{where}: a layer of type '{kind}' is not part of this architecture ({', '.join(sorted(mixers))})")
        norm = {"dim": self.width, "eps": self.eps}
        mlp, ffn, ffn_norm = _sub(layer, "mlp", where, needed=False), None, None
        if mlp is not None:
            ffn = self._mlp(mlp, where + " mlp")
            ffn_norm = PartSpec("rmsnorm", {**norm, "name": "norm2"})
        return LayerSpec(prefix=f"l{i}.", block="parallel_prenorm", mixer=mixers[kind](_sub(layer, "mixer", where), where + " mixer"),
                         mixer_norm=PartSpec("rmsnorm", {**norm, "name": "norm1"}), ffn=ffn, ffn_norm=ffn_norm,
                         options={"unused_norm": "norm2"} if ffn is None else {})

    def plan(self) -> ModelPlan:
        norm = {"dim": self.width, "eps": self.eps}
        return ModelPlan(
            hidden_size=self.width, vocab_size=self.vocab, max_positions=self.max_positions,
            embedding=PartSpec("embedding", {"vocab_size": self.vocab, "dim": self.width, "name": "embed"}),
            layers=tuple(self._layer(i, l) for i, l in enumerate(self.layers)),
            schedule=tuple(ScheduleEntry(i) for i in range(len(self.layers))),
            # (the logits' scale rides on the last norm's weight: the head is linear)
            final_norm=PartSpec("rmsnorm", {**norm, "name": "final.norm", "scale": self.logit_scale}),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "dim": self.width, "tied_to": None, "name": "head"}),
            stop_token_ids=(), bos_token_id=None,
        ).validate()
