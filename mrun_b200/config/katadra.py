"""Typed configuration of the Katadra decoder: layers whose sublayers read the residual stream itself
and whose outputs pass a layer norm (weight and bias) on their way into it.

Mixers (``layers[i].type``):

* ``parallel``: two mixers that read the same rows, summed with ``left_scale`` and ``right_scale``.
  *left* is a causal attention without rotation: q and k divided by their root mean square per
  head, a query temperature that grows with the position (``q_temp.coef``, ``q_temp.every``), a
  soft cap on the scores (``softcap``), a learned bias per distance bucket and head
  (``bias_max``), an output gate per feature; keys of ``dim`` and values of ``vdim`` features.
  *right* is a time mixing over shifted rows with a decay per head and key channel (``heads`` x
  ``dim``);
* ``mamba2``: a selective state-space mixer (``heads``, ``vdim``, ``state``, ``groups``, ``conv``,
  ``norm_groups``).

The feed-forward (``layers[i].mlp``, or null) is ``dense``: down(relu(up x)^2) of ``ff`` features.  A
layer with ``weights_of``: j runs layer j's weights with a cache and a state of its own.

config.json is nested: ``vocab``, ``width``, ``norm.eps``, ``layers``.  Two sizes are the shapes of
tensors and not in config.json: the rows of the bias table (``l<i>.mix.left.rel``) and the inner size
of the decay's low-rank projection (``l<i>.mix.right.w1``); a configuration made without a
checkpoint gives them as the keys ``bias_rows`` of the left and ``rank`` of the right mixer.
Checkpoint tensors are named ``embed``, ``head``, ``final.norm``, ``final.norm.b`` and
``l<i>.<part>`` without a ``.weight`` suffix.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .balivik import _number, checkpoint_shapes
from .base import ConfigError, eos_token_ids, req_int
from .spec import (DenseMLPSpec, GatedAttentionSpec, LayerNormSpec, LayerSpec, ModelSpec, ParallelMixerSpec,
                   ScheduleEntry, StateSpaceSpec, TimeMixingSpec)
from .zasesun import _count, _positive, _section


@dataclass(frozen=True)
class KatadraLayer:
    mixer: Any                       # ParallelMixerSpec | StateSpaceSpec
    feed_forward: Optional[Any]      # DenseMLPSpec | None
    weights_of: Optional[int]        # the layer whose weights this one runs (None: its own)
    raw: Any                         # the layer's entry of config.json, kept for to_dict()


def _from_shape(shapes: Mapping[str, tuple], tensor: str, m: Mapping[str, Any], key: str, where: str) -> int:
    """A size that is the first extent of a checkpoint tensor, or a key where there is no checkpoint."""
    if tensor in shapes and len(shapes[tensor]) == 2:
        return int(shapes[tensor][0])
    if m.get(key) is None:
        raise ConfigError(f"{where}{key}", f"is given neither by the checkpoint tensor {tensor} nor by the key")
    return _count(m, key, where)


@dataclass(frozen=True)
class KatadraConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[KatadraLayer, ...]
    max_positions: int = 1 << 20
    eos_token_id: Tuple[int, ...] = ()

    architecture = "Katadra"
    model_type = "katadra"

    # ------------------------------------------------------------------ reading
    @staticmethod
    def _attention(m: Mapping[str, Any], mw: str, prefix: str, width: int, eps: float, shapes: dict):
        heads = _count(m, "heads", mw)
        kv_heads = _count(m, "kv_heads", mw) if m.get("kv_heads") is not None else heads
        if heads % kv_heads:
            raise ConfigError(f"{mw}heads", f"({heads}) is not a multiple of kv_heads ({kv_heads})")
        dim = _count(m, "dim", mw)
        temp = None
        if m.get("q_temp") is not None:
            section = _section(m, "q_temp", mw)
            temp = (_number(section, "coef", f"{mw}q_temp."), _positive(section, "every", f"{mw}q_temp."))
        rows = _from_shape(shapes, f"{prefix}.rel", m, "bias_rows", mw)
        return GatedAttentionSpec(
            hidden=width, heads=heads, kv_heads=kv_heads, dim=dim,
            vdim=_count(m, "vdim", mw) if m.get("vdim") is not None else dim,
            softmax_scale=_positive(m, "scale", mw), eps=eps, qk_norm="unit", sink=False, head_gate=False,
            temperature=temp, soft_cap=_positive(m, "softcap", mw) if m.get("softcap") is not None else None,
            distance_bias=(rows, _positive(m, "bias_max", mw)), element_gate=True)

    @classmethod
    def _mixer(cls, i: int, layer: Mapping[str, Any], where: str, width: int, eps: float, shapes: dict):
        kind = layer.get("type")
        m = _section(layer, "mixer", where)
        mw = f"{where}mixer."
        if kind == "parallel":
            left = cls._attention(_section(m, "left", mw), f"{mw}left.", f"l{i}.mix.left", width, eps, shapes)
            r, rw = _section(m, "right", mw), f"{mw}right."
            right = TimeMixingSpec(hidden=width, heads=_count(r, "heads", rw), dim=_count(r, "dim", rw),
                                   rank=_from_shape(shapes, f"l{i}.mix.right.w1", r, "rank", rw), eps=eps)
            return ParallelMixerSpec(hidden=width, left=left, right=right, eps=eps, combine="sum",
                                     scales=(_number(m, "left_scale", mw), _number(m, "right_scale", mw)))
        if kind == "mamba2":
            heads, groups = _count(m, "heads", mw), _count(m, "groups", mw)
            if heads % groups:
                raise ConfigError(f"{mw}heads", f"({heads}) is not a multiple of groups ({groups})")
            vdim, parts = _count(m, "vdim", mw), _count(m, "norm_groups", mw)
            if heads * vdim % parts:
                raise ConfigError(f"{mw}norm_groups", f"({parts}) does not divide the {heads * vdim} inner features")
            return StateSpaceSpec(hidden=width, heads=heads, vdim=vdim, state=_count(m, "state", mw), groups=groups,
                                  conv=_count(m, "conv", mw), norm_groups=parts, eps=eps)
        raise ConfigError(f"{where}type", f"names the unknown mixer {kind!r}")

    @staticmethod
    def _feed_forward(layer: Mapping[str, Any], where: str, width: int):
        mlp = layer.get("mlp")
        if mlp is None:
            return None
        if not isinstance(mlp, dict):
            raise ConfigError(f"{where}mlp", "is neither an object nor null")
        if mlp.get("kind", "dense") != "dense":
            raise ConfigError(f"{where}mlp.kind", f"names the unknown feed-forward {mlp.get('kind')!r}")
        return DenseMLPSpec(hidden=width, intermediate=_count(mlp, "ff", f"{where}mlp."))

    @classmethod
    def from_dict(cls, cfg: Mapping[str, Any], model_dir: Optional[str] = None) -> "KatadraConfig":
        vocab, width = req_int(cfg, "vocab"), req_int(cfg, "width")
        eps = _positive(_section(cfg, "norm", ""), "eps", "norm.")
        entries = cfg.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("layers", "is missing or empty")
        for i, entry in enumerate(entries):
            if not isinstance(entry, dict):
                raise ConfigError(f"layers[{i}]", "is not an object")
        shapes = checkpoint_shapes(model_dir)
        layers = []
        for i, entry in enumerate(entries):
            owner = cls._owner(entries, i)
            where = f"layers[{owner}]."
            source = entries[owner]
            layers.append(KatadraLayer(cls._mixer(owner, source, where, width, eps, shapes),
                                       cls._feed_forward(source, where, width), owner if owner != i else None, entry))
        positions = cfg.get("max_positions")
        return cls(vocab=vocab, width=width, eps=eps, layers=tuple(layers),
                   max_positions=req_int(cfg, "max_positions") if positions is not None else 1 << 20,
                   eos_token_id=eos_token_ids(model_dir, cfg))

    @staticmethod
    def _owner(entries, i: int) -> int:
        """The layer whose weights layer i runs: itself, or the one its ``weights_of`` leads to."""
        at, seen = i, {i}
        while entries[at].get("weights_of") is not None:
            at = _count(entries[at], "weights_of", f"layers[{at}].", 0)
            if at >= len(entries):
                raise ConfigError(f"layers[{i}].weights_of", f"names layer {at} of {len(entries)}")
            if at in seen:
                raise ConfigError(f"layers[{i}].weights_of", "leads back to a layer that has no weights of its own")
            seen.add(at)
        return at

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
        norm = LayerNormSpec(self.width, self.eps, bare=True, bias=True)
        layers, at = [], {}         # at: layer number of config.json -> place among the layers with weights
        for i, layer in enumerate(self.layers):
            if layer.weights_of is not None:
                continue
            at[i] = len(layers)
            layers.append(LayerSpec(
                prefix=f"l{i}", mixer=layer.mixer, feed_forward=layer.feed_forward, mixer_norm=norm,
                feed_forward_norm=norm if layer.feed_forward is not None else None, arrangement="post_norm",
                mixer_prefix="mix", feed_forward_prefix="mlp", mixer_norm_prefix="norm1", feed_forward_norm_prefix="norm2"))
        schedule = tuple(ScheduleEntry(at[i if layer.weights_of is None else layer.weights_of])
                         for i, layer in enumerate(self.layers))
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width,
            max_positions=self.max_positions, layers=tuple(layers), final_norm=norm, tie_embeddings=False,
            schedule=schedule, embedding_name="embed", final_norm_prefix="final.norm", head_name="head",
            eos_token_ids=self.eos_token_id, ignored_prefixes=(), ignored_containing=())
