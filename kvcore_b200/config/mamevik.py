"""Typed reader of a Mamevik model folder's config.json, and its description as parts.

Mamevik is a pre-norm decoder on one 32-bit stream, ``x <- x + mixer(norm1(x))`` and then ``x <- x + ff(norm2(x))``,
whose norms are RMS norms with a weight stored around zero.  The stream starts as the normed sum of a token's row and
a row of a second table that the token and the one in front of it choose together; a run of layers is taken several
times with the same weights, each pass begun with ``x <- W [x; x_0] + step[pass]`` (``x_0``: what the stream started
as).  The head is the embedding table; the logits are scaled and bounded smoothly.  Its keys:

    architecture      "Mamevik"
    vocab, width      vocabulary and stream width
    norm.eps          eps of every norm of the model
    embedding.bigram  {buckets, mul_prev, mul_cur} of the second table (key absent: no second table)
    loop              {start, stop, times} (key absent: every layer once)
    logit_scale       factor on the logits
    logit_softcap     their bound (key absent: none)
    layers[i]         type ("mamba2" | "latent_attention"), mixer {...},
                      mlp (null | {kind "moe", expert {ff, limit}, router {experts, top}})

``mamba2``: the selective state-space mixer, mixer {heads, vdim, state, groups, conv, norm_groups}.
``latent_attention``: attention over one cached latent vector a token without positions, mixer {heads, dim, vdim,
kv_rank, scale, mask {size}} (mask absent: every earlier token is seen), with a sink a head.
The mixture of experts chooses by the logits (with a bias) and weights by the softmax over the chosen ones; an expert
is the bounded gated unit.

Tensors: ``embed``, ``bigram``, ``embed.norm``, ``loop.in``, ``loop.step``, ``final.norm``, ``l<i>.norm{1,2}``,
``l<i>.mix.{in,conv,conv.b,dt_bias,A_log,D,norm,o}`` (mamba2), ``l<i>.mix.{q,dkv,dkv.norm,uk,uv,sink,o}``
(latent_attention), ``l<i>.mlp.{router,router.b,e<j>.{gate,up,down}}``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from .config_json import ConfigError
from .model_spec import LayerSpec, ModelSpec, PartSpec, default_schedule, looped_schedule
from .toposun import DEFAULT_MAX_POSITIONS, _need, _number, _positive_int

ARCHITECTURE = "Mamevik"
# constants the design fixes
NORM_WEIGHT_OFFSET = 1.0                 # norms multiply by (1 + w)
EXPERT_ALPHA, EXPERT_SHIFT = 1.702, 1.0  # an expert: g sigmoid(alpha g) (u + shift)


def _whole(raw: Mapping[str, Any], key: str, where: str) -> int:
    value = _need(raw, key, where)
    if isinstance(value, bool) or not isinstance(value, int):
        raise ConfigError(f"config.json: {where}.{key} must be a whole number, got {value!r}")
    return value


@dataclass(frozen=True)
class MamevikConfig:
    vocab: int
    width: int
    eps: float
    bigram: Mapping[str, int] | None
    loop: tuple[int, int, int] | None        # start, stop, times
    logit_scale: float
    logit_softcap: float | None
    layers: tuple[Mapping[str, Any], ...]
    max_positions: int
    stored_dtype: str | None

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "MamevikConfig":
        layers = _need(raw, "layers", "the model")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: layers must be a non-empty list")
        for index, layer in enumerate(layers):
            if not isinstance(layer, Mapping):
                raise ConfigError(f"config.json: layers[{index}] is not an object")
        pair = (raw.get("embedding") or {}).get("bigram")
        if pair is not None:
            where = "embedding.bigram"
            pair = dict(buckets=_positive_int(pair, "buckets", where), mul_prev=_whole(pair, "mul_prev", where),
                        mul_cur=_whole(pair, "mul_cur", where))
        loop = raw.get("loop")
        if loop is not None:
            loop = (_whole(loop, "start", "loop"), _whole(loop, "stop", "loop"), _positive_int(loop, "times", "loop"))
            if not 0 <= loop[0] < loop[1] <= len(layers):
                raise ConfigError(f"config.json: loop over layers [{loop[0]}, {loop[1]}) of {len(layers)}")
        cap = _number(raw, "logit_softcap", "the model") if raw.get("logit_softcap") is not None else None
        if cap is not None and not cap > 0:
            raise ConfigError(f"config.json: logit_softcap must be positive, got {cap}")
        return cls(
            vocab=_positive_int(raw, "vocab", "the model"),
            width=_positive_int(raw, "width", "the model"),
            eps=_number(_need(raw, "norm", "the model"), "eps", "norm"),
            bigram=pair,
            loop=loop,
            logit_scale=_number(raw, "logit_scale", "the model") if "logit_scale" in raw else 1.0,
            logit_softcap=cap,
            layers=tuple(layers),
            max_positions=int(raw.get("max_position_embeddings", DEFAULT_MAX_POSITIONS)),
            stored_dtype=raw.get("dtype") or raw.get("torch_dtype"),
        )

    # ---- parts ---------------------------------------------------------------------------------
    def _norm(self, tensor: str) -> PartSpec:
        return PartSpec("rmsnorm_stream", dict(size=self.width, eps=self.eps, name=tensor, tensor=tensor,
                                               offset=NORM_WEIGHT_OFFSET))

    def _state_space(self, index: int, m: Mapping[str, Any]) -> PartSpec:
        where = f"layers[{index}].mixer"
        heads, groups = _positive_int(m, "heads", where), _positive_int(m, "groups", where)
        vdim, norm_groups = _positive_int(m, "vdim", where), _positive_int(m, "norm_groups", where)
        if heads % groups:
            raise ConfigError(f"config.json: {where}.heads {heads} is not a multiple of groups {groups}")
        if heads * vdim % norm_groups:
            raise ConfigError(f"config.json: {where}: {heads} x {vdim} values do not fall into norm_groups {norm_groups}")
        return PartSpec("selective_state_space", dict(
            hidden_size=self.width, num_heads=heads, num_groups=groups, state_dim=_positive_int(m, "state", where),
            value_dim=vdim, conv_taps=_positive_int(m, "conv", where), norm_groups=norm_groups, eps=self.eps,
            name=f"l{index}.mix"))

    def _attention(self, index: int, m: Mapping[str, Any]) -> PartSpec:
        where = f"layers[{index}].mixer"
        mask = m.get("mask")
        return PartSpec("latent_attention", dict(
            hidden_size=self.width, num_heads=_positive_int(m, "heads", where), head_dim=_positive_int(m, "dim", where),
            rot_dim=0, rot_dims=0, rot_base=1.0, value_dim=_positive_int(m, "vdim", where),
            kv_rank=_positive_int(m, "kv_rank", where), scale=_number(m, "scale", where), eps=self.eps, sink=True,
            gate=False, window=_positive_int(mask, "size", where + ".mask") if mask else None, name=f"l{index}.mix"))

    def _feed_forward(self, index: int, layer: Mapping[str, Any]) -> PartSpec | None:
        mlp = layer.get("mlp")
        if mlp is None:
            return None
        where, name = f"layers[{index}].mlp", f"l{index}.mlp"
        kind = _need(mlp, "kind", where)
        if kind != "moe":
            raise ConfigError(f"config.json: {where}.kind {kind!r} is not a feed-forward of this design")
        router, expert = _need(mlp, "router", where), _need(mlp, "expert", where)
        experts, top = _positive_int(router, "experts", where + ".router"), _positive_int(router, "top", where + ".router")
        if top > experts:
            raise ConfigError(f"config.json: {where}.router.top {top} exceeds experts {experts}")
        limit = _number(expert, "limit", where + ".expert")
        if not limit > 0:
            raise ConfigError(f"config.json: {where}.expert.limit must be positive, got {limit}")
        return PartSpec("routed_experts", dict(
            hidden_size=self.width, num_experts=experts, top_k=top, expert_size=_positive_int(expert, "ff", where + ".expert"),
            score="softmax_chosen", weight_on="output", router_bias=True, join=(EXPERT_ALPHA, limit, EXPERT_SHIFT),
            tensor_names={"router": "router", "router_bias": "router.b", "gate": "e{index}.gate", "up": "e{index}.up",
                          "down": "e{index}.down"},
            name=name))

    def to_model_spec(self) -> ModelSpec:
        layers = []
        for index, layer in enumerate(self.layers):
            kind = _need(layer, "type", f"layers[{index}]")
            m = _need(layer, "mixer", f"layers[{index}]")
            if kind == "mamba2":
                mixer = self._state_space(index, m)
            elif kind == "latent_attention":
                mixer = self._attention(index, m)
            else:
                raise ConfigError(f"config.json: layers[{index}].type {kind!r} is not a mixer of this design")
            feed_forward = self._feed_forward(index, layer)
            prefix = f"l{index}"
            norms = {"mixer_norm": self._norm(f"{prefix}.norm1")}
            block: dict[str, Any] = {}
            if feed_forward is not None:
                norms["feed_forward_norm"] = self._norm(f"{prefix}.norm2")
            else:                        # a layer without a feed-forward may still carry the norm in front of one
                block["unused_tensors"] = (f"{prefix}.norm2",)
            layers.append(LayerSpec(prefix=prefix, block=PartSpec("prenorm_stream", block), mixer=mixer,
                                    feed_forward=feed_forward, norms=norms))
        embedding: dict[str, Any] = dict(vocab_size=self.vocab, hidden_size=self.width, name="embed", tensor="embed",
                                         norm=dict(tensor="embed.norm", eps=self.eps, offset=NORM_WEIGHT_OFFSET))
        if self.bigram is not None:
            embedding["pairs"] = dict(self.bigram, tensor="bigram")
        schedule, steps = default_schedule(len(layers)), {}
        if self.loop is not None:
            start, stop, times = self.loop
            schedule = looped_schedule(len(layers), start, stop, times, step="loop")
            steps["loop"] = PartSpec("recall_origin", dict(hidden_size=self.width, times=times, in_tensor="loop.in",
                                                           step_tensor="loop.step"))
        return ModelSpec(
            architecture=ARCHITECTURE,
            vocab_size=self.vocab,
            hidden_size=self.width,
            layers=tuple(layers),
            schedule=schedule,
            embedding=PartSpec("token_embedding", embedding),
            final_norm=self._norm("final.norm"),
            lm_head=PartSpec("lm_head", dict(vocab_size=self.vocab, hidden_size=self.width, name="lm_head", tied_to="embed",
                                             logit_scale=self.logit_scale, softcap=self.logit_softcap)),
            max_position_embeddings=self.max_positions,
            stored_dtype=self.stored_dtype,
            stream_steps=steps,
        )


__all__ = ["ARCHITECTURE", "MamevikConfig"]
