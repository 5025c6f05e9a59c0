"""The Semadra decoder's configuration, from its own config.json keys.

config.json: `architecture` "Semadra", `vocab`, `width`, `norm.eps`, `embedding.scale` (absent: 1), `residual_mult` (absent: 1),
`token_side.dim` (absent: no token input in the layers) and `layers`, one entry per layer: `type` ("attention" or
"latent_attention"), `mixer` (its sizes and constants) and `mlp` (a dense or a mixture-of-experts feed-forward, or null for
none).  Optional: `max_positions`.  Tensors: `embed` (also the head), `side.embed`, `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.*`, `l<i>.mlp.*`,
`l<i>.side.{gate,proj,norm}`, `final.norm`.

The norms are on the sublayers' outputs (block "sublayer_norm"): with m = `residual_mult`, x += m norm1(mixer(x)); x += m norm2(ff(x));
x += m norm(token input).  Norm weights of the layers and the last norm are stored around zero (1 + w); the token input's is plain.
  attention          softmax attention without positions (`parts/masked_attention.py`): `heads`, `kv_heads`, `dim`, `vdim`, `scale`,
                     `mask` {size, keep_first} (a sliding window behind which the first tokens stay visible; absent: causal), queries and keys
                     normed over the whole projection, an output gate per channel
  latent_attention   attention over a shared latent without a rotated part (`parts/latent_attention.py`): `heads`, `dim`, `vdim`, `q_rank`
                     (the queries' latent; absent: the stored tensor's size), `kv_rank`, `scale`, `mask` {size} (a sliding window); with
                     `kv_from`: j it keeps nothing and reads layer j's latent
The feed-forward: {"kind": "dense", "ff"}: a gated unit with silu; {"kind": "moe", "expert": {ff}, "router": {experts, top, groups {count,
keep}, scale}, "shared": {ff}}: experts scored by a sigmoid each, chosen inside the groups whose two best scores sum highest, weighted with
their scores times `scale`; a shared expert is added as it is.  The token input: `parts/token_side.py`, layer i reading the columns
i dim .. (i + 1) dim - 1 of its table.
"""
import dataclasses
from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

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


@register_architecture("Semadra", model_type="semadra")
@dataclass(frozen=True)
class SemadraConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[Mapping[str, Any], ...]
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    side_dim: Optional[int] = None
    max_positions: int = DEFAULT_MAX_POSITIONS

    architecture = "Semadra"

    @classmethod
    def from_dict(cls, d):
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' should be a non-empty list")
        emb, side = _sub(d, "embedding", "config.json", needed=False), _sub(d, "token_side", "config.json", needed=False)
        cfg = cls(vocab=require(d, "vocab", int), width=require(d, "width", int),
                  eps=require(_sub(d, "norm", "config.json"), "eps", float, "config.json norm"), layers=tuple(layers),
                  embedding_scale=optional(emb, "scale", float, 1.0, "config.json embedding") if emb is not None else 1.0,
                  residual_mult=optional(d, "residual_mult", float, 1.0),
                  side_dim=require(side, "dim", int, "config.json token_side") if side is not None else None,
                  max_positions=optional(d, "max_positions", int, DEFAULT_MAX_POSITIONS))
        if cfg.vocab <= 0 or cfg.width <= 0 or cfg.max_positions <= 0 or not cfg.eps > 0:
            raise ConfigError("config.json: vocab, width, max_positions and norm.eps must be positive")
        cfg.plan()     # every layer's keys are read and checked here
        return cfg

    def to_dict(self):
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
               "embedding": {"scale": self.embedding_scale}, "residual_mult": self.residual_mult, "layers": [dict(l) for l in self.layers]}
        if self.side_dim is not None:
            out["token_side"] = {"dim": self.side_dim}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        return out

    def shape_given_sizes(self, shapes):
        """The same configuration with every latent query size that config.json leaves out taken from the stored tensor's shape."""
        layers = list(self.layers)
        for i, l in enumerate(layers):
            m, name = l.get("mixer"), f"l{i}.mix.dq"
            if l.get("type") == "latent_attention" and m.get("q_rank") is None and name in shapes:
                layers[i] = {**l, "mixer": {**m, "q_rank": int(shapes[name][0])}}
        return dataclasses.replace(self, layers=tuple(layers))

    # ------------------------------------------------------------------ mixers
    def _attention(self, m, where):
        heads, dim = require(m, "heads", int, where), require(m, "dim", int, where)
        mask = _sub(m, "mask", where, needed=False)
        return PartSpec("masked_attention", {
            "hidden_size": self.width, "num_heads": heads, "num_kv_heads": optional(m, "kv_heads", int, None, where) or heads,
            "head_dim": dim, "v_head_dim": optional(m, "vdim", int, None, where) or dim, "scale": require(m, "scale", float, where),
            "qk_norm": {"eps": self.eps, "over": "projection"}, "channel_gate": True,
            "mask": {"kind": "window", "size": require(mask, "size", int, where + " mask"),
                     "keep_first": optional(mask, "keep_first", int, 0, where + " mask")} if mask is not None else None,
            "names": {"q": "mix.q", "k": "mix.k", "v": "mix.v", "o": "mix.o", "q_norm": "mix.q.norm", "k_norm": "mix.k.norm", "gate": "mix.g"}})

    def _latent(self, i, m, where):
        kv_from, dim, mask = optional(m, "kv_from", int, None, where), require(m, "dim", int, where), _sub(m, "mask", where, needed=False)
        if kv_from is not None:
            src = self.layers[kv_from] if 0 <= kv_from < i and isinstance(self.layers[kv_from], Mapping) else None
            sm = src.get("mixer") if src is not None and src.get("type") == "latent_attention" else None
            if not isinstance(sm, Mapping) or sm.get("kv_from") is not None:
                raise ConfigError(f"{where}: kv_from {kv_from} should name an earlier latent_attention layer that keeps its own latent")
            if sm.get("kv_rank") != m.get("kv_rank"):
                raise ConfigError(f"{where}: layer {kv_from}'s kv_rank differs from this layer's")
        return PartSpec("latent_attention", {
            "hidden_size": self.width, "num_heads": require(m, "heads", int, where), "head_dim": dim, "rot_dim": 0,
            "v_head_dim": optional(m, "vdim", int, None, where) or dim, "kv_rank": require(m, "kv_rank", int, where),
            "q_rank": optional(m, "q_rank", int, 1, where),      # (left out: `shape_given_sizes` puts the stored size in its place)
            "scale": require(m, "scale", float, where), "eps": self.eps, "reads_cache": kv_from is not None,
            "mask": {"kind": "window", "size": require(mask, "size", int, where + " mask")} if mask is not None else None,
            "names": {"dq": "mix.dq", "dq_norm": "mix.dq.norm", "uq": "mix.uq", "dkv": "mix.dkv", "dkv_norm": "mix.dkv.norm", "uk": "mix.uk",
                      "uv": "mix.uv", "o": "mix.o"}}), kv_from

    # ------------------------------------------------------------------ feed-forwards
    def _gated(self, ff, prefix):
        return PartSpec("swiglu", {"hidden_size": self.width, "intermediate_size": ff,
                                   "names": {k: prefix + k for k in ("gate", "up", "down")}})

    def _mlp(self, mlp, where):
        kind = require(mlp, "kind", str, where)
        if kind == "dense":
            return self._gated(require(mlp, "ff", int, where), "mlp.")
        if kind != "moe":
            raise ConfigError(f"{where}: kind '{kind}' is not part of this architecture (dense, moe)")
        e, r, shared = _sub(mlp, "expert", where), _sub(mlp, "router", where), _sub(mlp, "shared", where, needed=False)
        groups, rw = _sub(r, "groups", where + " router", needed=False), where + " router groups"
        return PartSpec("moe", {
            "hidden_size": self.width, "intermediate_size": require(e, "ff", int, where + " expert"),
            "experts": require(r, "experts", int, where + " router"), "top": require(r, "top", int, where + " router"),
            "router": {"kind": "scored", "score": "sigmoid", "renormalize": False, "scale": optional(r, "scale", float, 1.0, where + " router"),
                       "groups": require(groups, "count", int, rw) if groups is not None else 1,
                       "keep": require(groups, "keep", int, rw) if groups is not None else 1, "group_score": "top2_sum"},
            "shared": self._gated(require(shared, "ff", int, where + " shared"), "mlp.shared.") if shared is not None else None,
            "names": {"expert": "mlp.e", "gate": "gate", "up": "up", "down": "down", "router": "mlp.router"}})

    def _layer(self, i, layer):
        where = f"config.json layers[{i}]"
        if not isinstance(layer, Mapping):
            raise ConfigError(f"{where} should be an object")
        kind, m, reads = require(layer, "type", str, where), _sub(layer, "mixer", where), None
        if kind == "attention":
            mixer = self._attention(m, where + " mixer")
        elif kind == "latent_attention":
            mixer, reads = self._latent(i, m, where + " mixer")
        else:
            raise ConfigError(f"{where}: a layer of type '{kind}' is not part of this architecture (attention, latent_attention)")
        # (the constant that every sublayer's normed output is multiplied by rides on its norm's weight)
        norm = {"dim": self.width, "eps": self.eps, "scale": self.residual_mult}
        mlp, ffn, ffn_norm, options = _sub(layer, "mlp", where, needed=False), None, None, {}
        if mlp is not None:
            ffn = self._mlp(mlp, where + " mlp")
            ffn_norm = PartSpec("rmsnorm", {**norm, "offset": 1.0, "name": "norm2"})
        else:
            options["unused_norm"] = "norm2"
        if self.side_dim is not None:
            side = PartSpec("token_side", {"hidden_size": self.width, "dim": self.side_dim, "vocab_size": self.vocab,
                                           "columns": self.side_dim * len(self.layers), "first_column": self.side_dim * i,
                                           "names": {"table": "side.embed", "gate": "side.gate", "proj": "side.proj"}})
            options["after"] = ((side, PartSpec("rmsnorm", {**norm, "name": "side.norm"})),)
        return LayerSpec(prefix=f"l{i}.", block="sublayer_norm", mixer=mixer, mixer_norm=PartSpec("rmsnorm", {**norm, "offset": 1.0, "name": "norm1"}),
                         ffn=ffn, ffn_norm=ffn_norm, options=options), reads

    def plan(self) -> ModelPlan:
        built = [self._layer(i, l) for i, l in enumerate(self.layers)]
        return ModelPlan(
            hidden_size=self.width, vocab_size=self.vocab, max_positions=self.max_positions,
            embedding=PartSpec("embedding", {"vocab_size": self.vocab, "dim": self.width, "name": "embed", "scale": self.embedding_scale}),
            layers=tuple(spec for spec, _ in built),
            schedule=tuple(ScheduleEntry(i, reads) for i, (_, reads) in enumerate(built)),     # (a layer runs once: entry i is layer i)
            final_norm=PartSpec("rmsnorm", {"dim": self.width, "eps": self.eps, "offset": 1.0, "name": "final.norm"}),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "dim": self.width, "tied_to": "embed", "name": "head"}),
            stop_token_ids=(), bos_token_id=None,
        ).validate()
