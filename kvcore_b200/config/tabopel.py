"""Typed reader of a Tabopel model folder's config.json, and its description as parts.

Tabopel is a decoder on one 32-bit stream with a norm on both sides of each sub-layer,
``x <- x + norm1b(mixer(norm1(x)))`` and then ``x <- x + norm2b(ff(norm2(x)))``; every norm is an RMS norm with a plain
weight.  The embedded tokens are multiplied by a constant; a run of layers is taken several times with the same weights,
each pass begun with ``x <- x + step[pass]``; the head is a matrix of its own.  Its keys:

    architecture     "Tabopel"
    vocab, width     vocabulary and stream width
    norm.eps         eps of every norm of the model
    embedding.scale  factor on the embedded tokens
    loop             {start, stop, times} (key absent: every layer once)
    layers[i]        type ("attention" | "attention_2" | "retention"), mixer {...},
                     mlp (null | {kind "dense", ff} | {kind "moe", expert {ff}, router {experts, top, identity}})

``attention``: grouped-query attention, mixer {heads, kv_heads, dim, vdim, scale, conv, rot {base, dims, scaling
{factor, low, high, original}}}; q, k and v pass a short causal convolution of ``conv`` taps, the first ``rot.dims``
entries of q and k turn in halves (with frequencies scaled by their wavelength where ``scaling`` is given), one is added
to the softmax's denominator, and the heads' output is multiplied by ``sigmoid(W_g h)`` entry by entry.
``attention_2``: the same with biases on q, k and v, an RMS norm over the whole q and the whole k projection ahead of the
rotation, scores bounded by ``softcap * tanh(score / softcap)``, a learned sink a head, and neither convolution nor gate.
``retention``: linear attention with one fixed decay a head, mixer {heads, dim, vdim, decay [heads], rot}; q and k turn, k
is multiplied by ``dim^(-1/2)``, every head's read-out is divided by its root mean square and multiplied by
``silu(W_g h)``.
Feed-forwards square the positive part between two products.  The mixture takes a softmax over all experts, chooses by
``score + correction`` and weights by the score; the last ``router.identity`` experts hand their input on.

Tensors: ``embed``, ``head``, ``loop.step``, ``final.norm``, ``l<i>.norm{1,1b,2,2b}``, ``l<i>.mix.{q,k,v,o}`` with
``{q,k,v}.conv, g`` (attention), ``{q,k,v}.b, {q,k}.norm, sink`` (attention_2) or ``g`` (retention),
``l<i>.mlp.{up,down}`` or ``l<i>.mlp.{router, correction, e<j>.{up,down}}``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from .config_json import ConfigError
from .mamevik import _whole
from .model_spec import LayerSpec, ModelSpec, PartSpec, default_schedule, looped_schedule
from .toposun import DEFAULT_MAX_POSITIONS, _need, _number, _positive_int

ARCHITECTURE = "Tabopel"
PLAIN_NAMES = {"up": "up", "down": "down"}


@dataclass(frozen=True)
class TabopelConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    loop: tuple[int, int, int] | None        # start, stop, times
    layers: tuple[Mapping[str, Any], ...]
    max_positions: int
    stored_dtype: str | None

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "TabopelConfig":
        layers = _need(raw, "layers", "the model")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: layers must be a non-empty list")
        for index, layer in enumerate(layers):
            if not isinstance(layer, Mapping):
                raise ConfigError(f"config.json: layers[{index}] is not an object")
        loop = raw.get("loop")
        if loop is not None:
            loop = (_whole(loop, "start", "loop"), _whole(loop, "stop", "loop"), _positive_int(loop, "times", "loop"))
            if not 0 <= loop[0] < loop[1] <= len(layers):
                raise ConfigError(f"config.json: loop over layers [{loop[0]}, {loop[1]}) of {len(layers)}")
        return cls(
            vocab=_positive_int(raw, "vocab", "the model"),
            width=_positive_int(raw, "width", "the model"),
            eps=_number(_need(raw, "norm", "the model"), "eps", "norm"),
            embedding_scale=_number(_need(raw, "embedding", "the model"), "scale", "embedding"),
            loop=loop,
            layers=tuple(layers),
            max_positions=int(raw.get("max_position_embeddings", DEFAULT_MAX_POSITIONS)),
            stored_dtype=raw.get("dtype") or raw.get("torch_dtype"),
        )

    # ---- parts ---------------------------------------------------------------------------------
    def _norm(self, tensor: str) -> PartSpec:
        return PartSpec("rmsnorm_stream", dict(size=self.width, eps=self.eps, name=tensor, tensor=tensor))

    def _rotation(self, m: Mapping[str, Any], dim: int, where: str) -> PartSpec | None:
        rot = m.get("rot")
        if not rot:
            return None
        where += ".rot"
        dims = _positive_int(rot, "dims", where, minimum=0)
        if dims % 2 or dims > dim:
            raise ConfigError(f"config.json: {where}.dims must be even and at most dim {dim}, got {dims}")
        if not dims:
            return None
        params = dict(head_dim=dim, rotary_dim=dims, theta=_number(rot, "base", where))
        scaling = rot.get("scaling")
        if scaling:
            where += ".scaling"
            low, high = _number(scaling, "low", where), _number(scaling, "high", where)
            factor, original = _number(scaling, "factor", where), _number(scaling, "original", where)
            if not (factor > 0 and original > 0 and 0 < low <= high):
                raise ConfigError(f"config.json: {where} needs a positive factor and original and 0 < low <= high")
            params.update(rope_type="llama3", factor=factor, low_freq_factor=low, high_freq_factor=high,
                          original_max_position_embeddings=original)
        return PartSpec("rope", params)

    def _attention(self, index: int, m: Mapping[str, Any], second: bool) -> PartSpec:
        where = f"layers[{index}].mixer"
        heads, kv_heads = _positive_int(m, "heads", where), _positive_int(m, "kv_heads", where)
        if heads % kv_heads:
            raise ConfigError(f"config.json: {where}.heads {heads} is not a multiple of kv_heads {kv_heads}")
        dim = _positive_int(m, "dim", where)
        cap = _number(m, "softcap", where) if second and m.get("softcap") is not None else None
        if cap is not None and not cap > 0:
            raise ConfigError(f"config.json: {where}.softcap must be positive, got {cap}")
        taps = _positive_int(m, "conv", where) if not second and m.get("conv") is not None else 0
        return PartSpec("grouped_attention", dict(
            hidden_size=self.width, num_heads=heads, num_kv_heads=kv_heads, head_dim=dim,
            value_dim=_positive_int(m, "vdim", where), scale=_number(m, "scale", where), eps=self.eps,
            position=self._rotation(m, dim, where), conv_taps=taps, bias=second, qk_norm=second, softcap=cap,
            sink="learned" if second else "one", gate=not second, name=f"l{index}.mix"))

    def _retention(self, index: int, m: Mapping[str, Any]) -> PartSpec:
        where = f"layers[{index}].mixer"
        heads, dim = _positive_int(m, "heads", where), _positive_int(m, "dim", where)
        decay = _need(m, "decay", where)
        if (not isinstance(decay, (list, tuple)) or len(decay) != heads
                or any(isinstance(a, bool) or not isinstance(a, (int, float)) or not 0.0 <= a < float("inf") for a in decay)):
            raise ConfigError(f"config.json: {where}.decay must be {heads} numbers that are not negative, one a head")
        return PartSpec("retention", dict(
            hidden_size=self.width, num_heads=heads, head_dim=dim, value_dim=_positive_int(m, "vdim", where),
            decay=tuple(float(a) for a in decay), eps=self.eps, position=self._rotation(m, dim, where),
            name=f"l{index}.mix"))

    def _feed_forward(self, index: int, layer: Mapping[str, Any]) -> PartSpec | None:
        mlp = layer.get("mlp")
        if mlp is None:
            return None
        where, name = f"layers[{index}].mlp", f"l{index}.mlp"
        kind = _need(mlp, "kind", where)
        if kind == "dense":
            return PartSpec("squared_relu", dict(hidden_size=self.width, intermediate_size=_positive_int(mlp, "ff", where),
                                                 tensor_names=PLAIN_NAMES, name=name))
        if kind != "moe":
            raise ConfigError(f"config.json: {where}.kind {kind!r} is not a feed-forward of this design")
        router, expert = _need(mlp, "router", where), _need(mlp, "expert", where)
        where += ".router"
        experts, top = _positive_int(router, "experts", where), _positive_int(router, "top", where)
        identity = _positive_int(router, "identity", where, minimum=0) if router.get("identity") is not None else 0
        if top > experts + identity:
            raise ConfigError(f"config.json: {where}.top {top} exceeds experts {experts} + identity {identity}")
        return PartSpec("routed_experts", dict(
            hidden_size=self.width, num_experts=experts, top_k=top,
            expert_size=_positive_int(expert, "ff", f"layers[{index}].mlp.expert"), score="softmax", renormalize=False,
            weight_on="output", choice_correction=True, identity_experts=identity, activation="squared_relu",
            tensor_names={"router": "router", "correction": "correction", "up": "e{index}.up", "down": "e{index}.down"},
            name=name))

    def to_model_spec(self) -> ModelSpec:
        layers = []
        for index, layer in enumerate(self.layers):
            kind = _need(layer, "type", f"layers[{index}]")
            m = _need(layer, "mixer", f"layers[{index}]")
            if kind == "retention":
                mixer = self._retention(index, m)
            elif kind in ("attention", "attention_2"):
                mixer = self._attention(index, m, kind == "attention_2")
            else:
                raise ConfigError(f"config.json: layers[{index}].type {kind!r} is not a mixer of this design")
            feed_forward = self._feed_forward(index, layer)
            prefix = f"l{index}"
            norms = {"mixer_norm": self._norm(f"{prefix}.norm1"), "mixer_out_norm": self._norm(f"{prefix}.norm1b")}
            block: dict[str, Any] = {}
            if feed_forward is not None:
                norms["feed_forward_norm"] = self._norm(f"{prefix}.norm2")
                norms["feed_forward_out_norm"] = self._norm(f"{prefix}.norm2b")
            else:                        # a layer without a feed-forward may still carry the norms around one
                block["unused_tensors"] = (f"{prefix}.norm2", f"{prefix}.norm2b")
            layers.append(LayerSpec(prefix=prefix, block=PartSpec("sandwich_stream", block), mixer=mixer,
                                    feed_forward=feed_forward, norms=norms))
        schedule, steps = default_schedule(len(layers)), {}
        if self.loop is not None:
            start, stop, times = self.loop
            schedule = looped_schedule(len(layers), start, stop, times, step="loop")
            steps["loop"] = PartSpec("add_step", dict(hidden_size=self.width, times=times, step_tensor="loop.step"))
        return ModelSpec(
            architecture=ARCHITECTURE,
            vocab_size=self.vocab,
            hidden_size=self.width,
            layers=tuple(layers),
            schedule=schedule,
            embedding=PartSpec("token_embedding", dict(vocab_size=self.vocab, hidden_size=self.width, name="embed",
                                                       tensor="embed", scale=self.embedding_scale)),
            final_norm=self._norm("final.norm"),
            lm_head=PartSpec("lm_head", dict(vocab_size=self.vocab, hidden_size=self.width, name="head", tensor="head")),
            max_position_embeddings=self.max_positions,
            stored_dtype=self.stored_dtype,
            stream_steps=steps,
        )


__all__ = ["ARCHITECTURE", "TabopelConfig"]
