"""Typed configuration of the Sebevik decoder: pre-norm layers, each with one of three mixers, over norms whose
weights are stored around zero and an embedding table that is the output head too.

Mixers (``layers[i].type``):

* ``latent_attention``: causal attention without positions whose keys and values are up-projections of
  one cached latent a token (``heads``, ``dim``, ``vdim``, ``kv_rank``, ``scale``), with an output gate per head;
* ``attention``: grouped-query attention over a sliding window (``mask.size``) with projection biases,
  interleaved rotary positions on the first ``rot.dims`` features (``rot.base``), q and k divided by their
  root mean square per head, a learned sink per head; layers with ``v_mix`` blend their values with those
  of the first such layer;
* ``mamba1``: a selective state-space mixer with a decay per channel and state (``inner``, ``state``, ``dt_rank``,
  ``conv``).

The feed-forward (``layers[i].mlp``, or null) is ``dense``: down(relu(up x)^2) of ``ff`` features, or ``moe``: gated
experts (``expert.ff``) behind a softmax router (``router``: ``experts``, ``top``, ``groups.count``, ``groups.keep``,
``identity``) with a correction for the choice, groups ranked by their best expert, identity experts and
weights that are not renormalized, beside a gated shared expert (``shared.ff``).

config.json is nested: ``vocab``, ``width``, ``norm.eps``, ``layers``.  Checkpoint tensors are named ``embed``,
``final.norm`` and ``l<i>.<part>`` without a ``.weight`` suffix.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .base import ConfigError, eos_token_ids, req_int
from .spec import (DenseMLPSpec, GatedAttentionSpec, GroupedRoutedMLPSpec, LatentAttentionSpec, LayerSpec, ModelSpec,
                   RMSNormSpec, ScaledRotarySpec, SelectiveScanSpec)
from .zasesun import _count, _positive, _section


@dataclass(frozen=True)
class SebevikLayer:
    mixer: Any                       # LatentAttentionSpec | GatedAttentionSpec | SelectiveScanSpec
    feed_forward: Optional[Any]      # DenseMLPSpec | GroupedRoutedMLPSpec | None
    raw: Any                         # the layer's entry of config.json, kept for to_dict()


@dataclass(frozen=True)
class SebevikConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[SebevikLayer, ...]
    max_positions: int = 1 << 20
    eos_token_id: Tuple[int, ...] = ()

    architecture = "Sebevik"
    model_type = "sebevik"

    # ------------------------------------------------------------------ reading
    @staticmethod
    def _rotary(m: Mapping[str, Any], mw: str, dim: int) -> Optional[ScaledRotarySpec]:
        if m.get("rot") is None:
            return None
        rot = _section(m, "rot", mw)
        dims = _count(rot, "dims", f"{mw}rot.", 0)
        if dims == 0:
            return None
        if dims % 2 or dims > dim:
            raise ConfigError(f"{mw}rot.dims", f"must be even and at most dim={dim}, got {dims}")
        return ScaledRotarySpec(dims=dims, base=_positive(rot, "base", f"{mw}rot."), pairing="interleaved")

    @classmethod
    def _attention(cls, m: Mapping[str, Any], mw: str, width: int, eps: float, first) -> GatedAttentionSpec:
        """``first``: the spec of the first layer that mixes values, None before it."""
        heads = _count(m, "heads", mw)
        kv_heads = _count(m, "kv_heads", mw) if m.get("kv_heads") is not None else heads
        if heads % kv_heads:
            raise ConfigError(f"{mw}heads", f"({heads}) is not a multiple of kv_heads ({kv_heads})")
        dim = _count(m, "dim", mw)
        vdim = _count(m, "vdim", mw) if m.get("vdim") is not None else dim
        mixes = m.get("v_mix")
        if mixes is not None and not isinstance(mixes, bool):
            raise ConfigError(f"{mw}v_mix", f"must be true or false, got {mixes!r}")
        if mixes and first is not None and (first.kv_heads, first.vdim) != (kv_heads, vdim):
            raise ConfigError(f"{mw}v_mix", f"blends values of {kv_heads} x {vdim} with those of the first such layer, "
                                            f"{first.kv_heads} x {first.vdim}")
        window = None
        if m.get("mask") is not None:
            window = _count(_section(m, "mask", mw), "size", f"{mw}mask.")
        return GatedAttentionSpec(
            hidden=width, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, softmax_scale=_positive(m, "scale", mw), eps=eps,
            qk_norm="unit", sink=True, head_gate=False, position=cls._rotary(m, mw, dim), window=window, biases=True,
            learned_sink=True, value_mix=None if not mixes else "first" if first is None else "blend")

    @classmethod
    def _mixer(cls, layer: Mapping[str, Any], where: str, width: int, eps: float, first):
        kind = layer.get("type")
        m = _section(layer, "mixer", where)
        mw = f"{where}mixer."
        if kind == "latent_attention":
            dim = _count(m, "dim", mw)
            return LatentAttentionSpec(hidden=width, heads=_count(m, "heads", mw), dim=dim, rot_dim=0,
                                       vdim=_count(m, "vdim", mw) if m.get("vdim") is not None else dim, q_rank=0,
                                       kv_rank=_count(m, "kv_rank", mw), softmax_scale=_positive(m, "scale", mw), eps=eps,
                                       head_gate=True)
        if kind == "attention":
            return cls._attention(m, mw, width, eps, first)
        if kind == "mamba1":
            return SelectiveScanSpec(hidden=width, inner=_count(m, "inner", mw), state=_count(m, "state", mw),
                                     dt_rank=_count(m, "dt_rank", mw), conv=_count(m, "conv", mw))
        raise ConfigError(f"{where}type", f"names the unknown mixer {kind!r}")

    @staticmethod
    def _feed_forward(layer: Mapping[str, Any], where: str, width: int):
        mlp = layer.get("mlp")
        if mlp is None:
            return None
        if not isinstance(mlp, dict):
            raise ConfigError(f"{where}mlp", "is neither an object nor null")
        fw = f"{where}mlp."
        kind = mlp.get("kind")
        if kind is None:        # left out: what the entry holds says which it is
            kind = "moe" if "router" in mlp else "dense" if "ff" in mlp else None
        if kind == "dense":
            return DenseMLPSpec(hidden=width, intermediate=_count(mlp, "ff", fw))
        if kind != "moe":
            raise ConfigError(f"{fw}kind", f"names the unknown feed-forward {kind!r}")
        router = _section(mlp, "router", fw)
        rw = f"{fw}router."
        experts, top = _count(router, "experts", rw), _count(router, "top", rw)
        identity = _count(router, "identity", rw, 0) if router.get("identity") is not None else 0
        groups = keep = 1
        if router.get("groups") is not None:
            section = _section(router, "groups", rw)
            groups, keep = _count(section, "count", f"{rw}groups."), _count(section, "keep", f"{rw}groups.")
            if (experts + identity) % groups:
                raise ConfigError(f"{rw}groups.count", f"({groups}) does not divide the {experts} + {identity} experts")
            if keep > groups:
                raise ConfigError(f"{rw}groups.keep", f"({keep}) exceeds the {groups} groups")
        allowed = keep * ((experts + identity) // groups)
        if top > allowed:
            raise ConfigError(f"{rw}top", f"({top}) exceeds the {allowed} experts that can be chosen")
        shared_ff = 0
        if mlp.get("shared") is not None:
            shared_ff = _count(_section(mlp, "shared", fw), "ff", f"{fw}shared.")
        return GroupedRoutedMLPSpec(hidden=width, experts=experts, top=top,
                                    expert_ff=_count(_section(mlp, "expert", fw), "ff", f"{fw}expert."), groups=groups,
                                    keep_groups=keep, group_top=1, shared_ff=shared_ff, shared_gate=True, score="softmax",
                                    correction=True, identity=identity, renormalize=False)

    @classmethod
    def from_dict(cls, cfg: Mapping[str, Any], model_dir: Optional[str] = None) -> "SebevikConfig":
        vocab, width = req_int(cfg, "vocab"), req_int(cfg, "width")
        eps = _positive(_section(cfg, "norm", ""), "eps", "norm.")
        entries = cfg.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("layers", "is missing or empty")
        layers, first = [], None
        for i, entry in enumerate(entries):
            where = f"layers[{i}]."
            if not isinstance(entry, dict):
                raise ConfigError(f"layers[{i}]", "is not an object")
            mixer = cls._mixer(entry, where, width, eps, first)
            if first is None and getattr(mixer, "value_mix", None) is not None:
                first = mixer
            layers.append(SebevikLayer(mixer, cls._feed_forward(entry, where, width), entry))
        positions = cfg.get("max_positions")
        return cls(vocab=vocab, width=width, eps=eps, layers=tuple(layers),
                   max_positions=req_int(cfg, "max_positions") if positions is not None else 1 << 20,
                   eos_token_id=eos_token_ids(model_dir, cfg))

    def to_dict(self) -> dict:
        """config.json contents that :meth:`from_dict` reads back to an equal configuration."""
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
               "layers": [layer.raw for layer in self.layers]}
        if self.max_positions != 1 << 20:
            out["max_positions"] = self.max_positions
        if self.eos_token_id:
            out["eos_token_id"] = list(self.eos_token_id)
        return out

    # ------------------------------------------------------------------ derived
    def num_parameters(self) -> int:
        from ..weights.loader import expected_tensors
        total = 0
        for t in expected_tensors(self.to_spec()):
            count = 1
            for extent in t.shape:
                count *= extent
            total += count
        return total

    def to_spec(self) -> ModelSpec:
        norm = RMSNormSpec(self.width, self.eps, bare=True, offset=1.0)
        layers = tuple(
            LayerSpec(prefix=f"l{i}", mixer=layer.mixer, feed_forward=layer.feed_forward, mixer_norm=norm,
                      feed_forward_norm=norm if layer.feed_forward is not None else None, arrangement="pre_norm",
                      mixer_prefix="mix", feed_forward_prefix="mlp", mixer_norm_prefix="norm1",
                      feed_forward_norm_prefix="norm2")
            for i, layer in enumerate(self.layers))
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width,
            max_positions=self.max_positions, layers=layers, final_norm=norm, tie_embeddings=True, embedding_name="embed",
            final_norm_prefix="final.norm", eos_token_ids=self.eos_token_id, ignored_prefixes=(), ignored_containing=())
