"""Typed configuration of Tudulix, read from its own config.json keys.

A Tudulix folder names itself with ``"architecture": "Tudulix"`` and gives ``vocab``, ``width``, ``norm.eps``,
``embedding.scale``, ``logit_scale``, a list ``layers`` and, where layers run more than once, ``loop``; every layer has a
``type`` (which mixer), the mixer's sizes and constants under ``mixer`` and its feed-forward under ``mlp`` (``null``: none).
Layers are parsed one by one: nothing is assumed about their number, order or sizes.

Two mixers exist.  ``attention`` is grouped-query attention over a window.  ``latent_attention`` attends, over a window as
well, through one cached latent per token.  The feed-forward is ``moe``: routed experts and, where ``mlp.shared`` is given,
one more expert that runs for every token, with a size and a limit of its own.  ``loop`` runs the layers ``start`` ..
``stop`` - 1 ``times`` times in a row with the same weights, which maps onto run-order entries that name a block more than
once: every pass has caches of its own, and the embedding's output joins the stream before every pass but the first.

What the design fixes, and what this file therefore writes down: an RMS norm before and after each sublayer, its scale
stored around zero; the attention pairs adjacent elements of a head, the latent attention the halves of its rotated
part; queries come from the input directly; a gate per element multiplies the latent attention's output; the unit inside an
expert is the clamped one with the constant 1.702; the router's logits carry a bias, and the weights are the softmax over the
chosen logits; the head is not tied and its logits are scaled; and the tensor names (``embed``, ``head``, ``final.norm``,
``l<i>.norm1`` / ``norm1b`` / ``norm2`` / ``norm2b``, ``l<i>.mix.*``, ``l<i>.mlp.*``).
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Optional, Tuple

from .reader import _Reader, _is_int
from .registry import ConfigError, extract_eos_token_ids, register_architecture
from .spec import (BlockSpec, GqaSpec, LatentAttentionSpec, LayerCall, LinearHeadSpec, ModelSpec, NormSpec, RotaryRatesSpec,
                   RoutedExpertsSpec, ScaledEmbeddingSpec, looped_order)

UNIT_ALPHA = 1.702
MAX_POSITIONS = 1 << 20          # the design names no longest sequence; this bounds positions, not the arithmetic


def _window(m: _Reader) -> Optional[int]:
    return m.obj("mask").positive_int("size") if m.raw.get("mask") is not None else None


def _rotary(m: _Reader, adjacent: bool) -> RotaryRatesSpec:
    rot = m.obj("rot")
    dims = rot.positive_int("dims")
    if dims % 2:
        m.problems.append(f"{rot.where}: `dims`={dims} must be even")
    return RotaryRatesSpec(dims=dims, base=rot.number("base", positive=True), adjacent=adjacent)


def _attention(m: _Reader, width: int) -> GqaSpec:
    heads, kv_heads, dim = m.positive_int("heads"), m.positive_int("kv_heads"), m.positive_int("dim")
    if heads % kv_heads:
        m.problems.append(f"{m.where}: heads={heads} is not a multiple of kv_heads={kv_heads}")
    position = _rotary(m, True)
    if position.dims > dim:
        m.problems.append(f"{m.where}.rot: `dims`={position.dims} must be at most the {dim} elements of a head")
    return GqaSpec(hidden_size=width, num_heads=heads, num_kv_heads=kv_heads, head_dim=dim, value_dim=m.positive_int("vdim"),
                   softmax_scale=m.number("scale", positive=True), position=position, window=_window(m))


def _latent_attention(m: _Reader, width: int, eps: float) -> LatentAttentionSpec:
    rot_dim = m.positive_int("rot_dim")
    position = _rotary(m, False)
    if position.dims > rot_dim:
        m.problems.append(f"{m.where}.rot: `dims`={position.dims} must be at most the {rot_dim} elements it turns")
    return LatentAttentionSpec(hidden_size=width, num_heads=m.positive_int("heads"), head_dim=m.positive_int("dim"), rot_dim=rot_dim,
                               value_dim=m.positive_int("vdim"), kv_rank=m.positive_int("kv_rank"), q_rank=None,
                               softmax_scale=m.number("scale", positive=True), norm_eps=eps, position=position, window=_window(m),
                               element_gate=True)


def _experts(f: _Reader, width: int) -> Optional[RoutedExpertsSpec]:
    if f.raw.get("kind") != "moe":
        f.problems.append(f"{f.where}: unknown kind {f.raw.get('kind')!r}; known: ['moe']")
        return None
    r, e = f.obj("router"), f.obj("expert")
    experts, top = r.positive_int("experts"), r.positive_int("top")
    if top > experts:
        f.problems.append(f"{r.where}: top={top} of {experts} experts")
    shared_size, shared_limit = None, 0.0
    if f.raw.get("shared") is not None:
        sh = f.obj("shared")
        shared_size, shared_limit = sh.positive_int("ff"), sh.number("limit", positive=True)
    return RoutedExpertsSpec(hidden_size=width, expert_size=e.positive_int("ff"), n_experts=experts, top_k=min(top, experts),
                             scoring="softmax_chosen", activation="clamped_glu", limit=e.number("limit", positive=True), alpha=UNIT_ALPHA,
                             shared_size=shared_size, shared_limit=shared_limit, router_bias_name="router.b")


@register_architecture("Tudulix", aliases=("Tudulix", "TudulixModel"), model_types=("tudulix",))
@dataclass(frozen=True)
class TudulixConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    logit_scale: float
    blocks: Tuple[BlockSpec, ...]
    order: Tuple[LayerCall, ...]
    eos_token_ids: Tuple[int, ...] = ()
    raw: Optional[dict] = None

    @classmethod
    def from_dict(cls, raw: dict) -> "TudulixConfig":
        problems: list = []
        top = _Reader(raw, "config", problems)
        vocab, width = top.positive_int("vocab"), top.positive_int("width")
        eps = top.obj("norm").number("eps", positive=True)
        embedding_scale, logit_scale = top.obj("embedding").number("scale"), top.number("logit_scale")
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            problems.append("config: `layers` must be a non-empty list")
            layers = []
        norm = NormSpec(dim=width, eps=eps, suffix="", offset=1.0)
        blocks: list = []
        for i, layer in enumerate(layers):
            rd = _Reader(layer, f"layers[{i}]", problems)
            kind = rd.raw.get("type")
            m = rd.obj("mixer")
            mixer = None
            if kind == "attention":
                mixer = _attention(m, width)
            elif kind == "latent_attention":
                mixer = _latent_attention(m, width, eps)
            else:
                problems.append(f"layers[{i}]: unknown layer type {kind!r}; known: ['attention', 'latent_attention']")
            ff = None
            if rd.raw.get("mlp") is not None:
                ff = _experts(_Reader(rd.raw["mlp"], f"layers[{i}].mlp", problems), width)
            blocks.append(BlockSpec(mixer=mixer, feed_forward=ff, mixer_norm=norm, ff_norm=norm if ff is not None else None,
                                    prefix=f"l{i}", mixer_name="mix", ff_name="mlp", mixer_norm_name="norm1", ff_norm_name="norm2",
                                    kind="sandwich_residual", mixer_post_norm=norm, ff_post_norm=norm if ff is not None else None,
                                    mixer_post_norm_name="norm1b", ff_post_norm_name="norm2b"))
        order = cls._order(raw.get("loop"), len(blocks), problems)
        try:
            eos = extract_eos_token_ids(raw)
        except ConfigError as e:
            problems.append(str(e))
            eos = ()
        if problems:
            raise ConfigError("failed to parse Tudulix config: " + "; ".join(problems))
        return cls(vocab=vocab, width=width, norm_eps=eps, embedding_scale=embedding_scale, logit_scale=logit_scale, blocks=tuple(blocks),
                   order=order, eos_token_ids=eos, raw=copy.deepcopy(raw))

    @staticmethod
    def _order(loop, n: int, problems: list) -> Tuple[LayerCall, ...]:
        plain = tuple(LayerCall(block=i) for i in range(n))
        if loop is None:
            return plain
        rd = _Reader(loop, "config.loop", problems)
        before = len(problems)
        start = rd.raw.get("start")
        if not _is_int(start) or start < 0:
            problems.append(f"config.loop: `start` must be the number of a layer, got {start!r}")
        stop, times = rd.positive_int("stop"), rd.positive_int("times")
        if len(problems) > before:
            return plain
        if not start < stop <= n:
            problems.append(f"config.loop: layers {start} .. {stop - 1} are not layers of {n}")
            return plain
        return looped_order(n, start, stop, times)

    def to_dict(self) -> dict:
        return copy.deepcopy(self.raw)

    def to_model_spec(self) -> ModelSpec:
        # a layer without a feed-forward reads no norms around it; a folder may carry them all the same
        unread = tuple(f"{b.prefix}.{name}" for b in self.blocks if b.feed_forward is None for name in ("norm2", "norm2b"))
        # the scale of the logits is the last norm's gain: the head between them is linear
        final = NormSpec(dim=self.width, eps=self.norm_eps, suffix="", offset=1.0, gain=self.logit_scale)
        return ModelSpec(architecture="Tudulix", vocab_size=self.vocab, hidden_size=self.width, max_positions=MAX_POSITIONS,
                         blocks=self.blocks, order=self.order, final_norm=final, tie_embeddings=False, embed_name="embed",
                         final_norm_name="final.norm", head_name="head", eos_token_ids=self.eos_token_ids,
                         embedding=ScaledEmbeddingSpec(self.vocab, self.width, self.embedding_scale, name="embed"),
                         head=LinearHeadSpec(self.vocab, self.width, tied=False, name="head"), ignored_tensors=unread)
