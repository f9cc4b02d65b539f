"""Grouped-query attention whose key and value widths differ, with its mechanisms as parameters.

    q, k, v = W_q x (+ b), W_k x (+ b), W_v x (+ b)                     (``bias``)
    each channel of q, k and v passes a causal convolution over time    (``conv_taps``: their number; 0: none)
    q and k: one RMS norm over the whole projection each, with weights  (``qk_norm``)
    q and k turn by the token's position                                (``position``: an encoding that offers its table)
    score = q . k * scale, then softcap * tanh(score / softcap)         (``softcap``)
    weight = exp(score) / (sink + sum exp(score)), every earlier token seen, with ``sink`` None: 0 (ordinary softmax);
             "one": 1; "learned": exp of one number a head
    o = sum of weights times values, times sigmoid(W_g x)               (``gate``: entry by entry)

A token's keys and values are one cached row ``[k of all kv heads | v of all kv heads]``; where both widths are the one
that the TMA decode and the tcgen05 prompt kernels are made for (bfloat16), they are the two planes of those kernels
instead (``CacheSpec.keys_and_values``).  With a convolution the last
``conv_taps - 1`` projected q, k and v of a request are per-request state (``[taps - 1, channels]``, 32-bit, oldest
first).  Scores, softmax, angles, norms and the convolution's sums are 32-bit whatever the activation type.
"""
from __future__ import annotations

import torch

from .. import kernels as K
from ..config.model_spec import PartSpec
from .base import MIXERS, POSITION_ENCODINGS, CacheSpec, StateSpec, WeightSlot
from .recurrent import ProjectedMixer, _round4, _round8


class GroupedAttention(ProjectedMixer):
    DEFAULT_TENSOR_NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "q_bias": "q.b", "k_bias": "k.b",
                            "v_bias": "v.b", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv",
                            "q_norm": "q.norm", "k_norm": "k.norm", "sink": "sink"}

    def __init__(self, *, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, value_dim: int,
                 scale: float, eps: float, name: str, position: PartSpec | None = None, conv_taps: int = 0,
                 bias: bool = False, qk_norm: bool = False, softcap: float | None = None, sink: str | None = None,
                 gate: bool = False, tensor_names: dict | None = None, dtype: torch.dtype, device: torch.device) -> None:
        if min(num_heads, num_kv_heads, head_dim, value_dim) <= 0 or num_heads % num_kv_heads:
            raise ValueError(f"num_heads {num_heads} must be a positive multiple of num_kv_heads {num_kv_heads}")
        if value_dim > 512:
            raise ValueError(f"value_dim {value_dim} exceeds the attention kernels' value width of 512")
        if softcap is not None and not softcap > 0:
            raise ValueError(f"the scores' cap must be positive, got {softcap}")
        if sink not in (None, "one", "learned"):
            raise ValueError(f"sink is None, 'one' or 'learned', got {sink!r}")
        if conv_taps < 0:
            raise ValueError(f"the convolution's taps are not negative, got {conv_taps}")
        self.hidden_size, self.num_heads, self.num_kv_heads = int(hidden_size), int(num_heads), int(num_kv_heads)
        self.head_dim, self.value_dim = int(head_dim), int(value_dim)
        self.scale, self.eps, self.name = float(scale), float(eps), name
        self.softcap = None if softcap is None else float(softcap)
        self.conv_taps, self.qk_norm, self.has_gate = int(conv_taps), bool(qk_norm), bool(gate)
        self.tensor_names = dict(self.DEFAULT_TENSOR_NAMES)
        self.tensor_names.update(tensor_names or {})
        self.q_cols = self.num_heads * self.head_dim
        self.k_cols = self.num_kv_heads * self.head_dim
        self.v_cols = self.num_kv_heads * self.value_dim
        # one packed projection: q, k, v, then (on a boundary of 8) the gate
        self.channels = self.q_cols + self.k_cols + self.v_cols
        self.out_cols = self.num_heads * self.value_dim
        self.g_col = _round8(self.channels)
        self.in_rows = _round8(self.g_col + (self.out_cols if self.has_gate else 0))
        self._allocate(dtype, device)
        on_device = dict(dtype=dtype, device=device)
        self.position = None if position is None else POSITION_ENCODINGS.build(position, dtype=dtype, device=device)
        if self.position is not None and getattr(self.position, "rotary_dim", 0) > self.head_dim:
            raise ValueError(f"{self.name}: the encoding turns more than a head's {self.head_dim} entries")
        self.in_bias = torch.zeros(self.in_rows, **on_device) if bias else None
        # taps as [taps, channels]: neighbouring channels' taps lie together
        self.taps = torch.empty(self.conv_taps, self.channels, **on_device) if self.conv_taps else None
        self.q_norm_weight = torch.empty(self.q_cols, **on_device) if self.qk_norm else None
        self.k_norm_weight = torch.empty(self.k_cols, **on_device) if self.qk_norm else None
        self.learned_sink = sink == "learned"
        self.sink = None
        if sink is not None:      # the logits that join the softmax's denominator: exp(0) adds one
            self.sink = torch.zeros(self.num_heads, dtype=torch.float32, device=device)

    @property
    def graph_safe(self) -> bool:
        return self.position is None or self.position.graph_safe

    # the page sizes of a cache do not count here: with one that those kernels do not take the planes are read by strides
    def _two_planes(self) -> bool:
        return self.head_dim == self.value_dim and K.paged_attention_takes_sinks(self.dtype, self.head_dim, 16)

    def cache_spec(self) -> CacheSpec:
        if self._two_planes():
            return CacheSpec.keys_and_values(self.num_kv_heads, self.head_dim)
        return CacheSpec(1, 1, self.k_cols + self.v_cols)

    def state_spec(self) -> StateSpec | None:
        if self.conv_taps < 2:
            return None
        return StateSpec((_round4(self.channels * (self.conv_taps - 1)),), torch.float32)

    def _tensor(self, key: str) -> str:
        return f"{self.name}.{self.tensor_names[key]}"

    def weight_slots(self) -> list[WeightSlot]:
        w = self.in_weight
        cuts = {"q": (0, self.q_cols), "k": (self.q_cols, self.q_cols + self.k_cols),
                "v": (self.q_cols + self.k_cols, self.channels)}
        slots = [WeightSlot(self._tensor(key), w[lo:hi]) for key, (lo, hi) in cuts.items()]
        slots.append(WeightSlot(self._tensor("o"), self.o_weight))
        if self.has_gate:
            slots.append(WeightSlot(self._tensor("g"), w[self.g_col:self.g_col + self.out_cols]))
        if self.in_bias is not None:
            slots += [WeightSlot(self._tensor(f"{key}_bias"), self.in_bias[lo:hi]) for key, (lo, hi) in cuts.items()]
        if self.taps is not None:
            slots += [WeightSlot(self._tensor(f"{key}_conv"), self.taps[:, lo:hi].t(), file_shape=(hi - lo, self.conv_taps))
                      for key, (lo, hi) in cuts.items()]
        if self.qk_norm:
            slots += [WeightSlot(self._tensor("q_norm"), self.q_norm_weight, init="ones"),
                      WeightSlot(self._tensor("k_norm"), self.k_norm_weight, init="ones")]
        if self.learned_sink:
            slots.append(WeightSlot(self._tensor("sink"), self.sink, init="zeros"))
        return slots

    def ignorable_tensor_names(self) -> list[str]:
        return [] if self.position is None else self.position.ignorable_tensor_names()

    def mix_rows(self, rows, ctx, cache, out, scale: float = 1.0) -> None:
        if scale != 1.0:
            raise ValueError(f"{self.name}: grouped attention writes its output without a factor")
        tokens, heads = rows.shape[0], self.num_heads
        table = ctx.block_table(cache.group)
        cos_sin = None
        if self.position is not None:
            cos_sin = self.position.cos_sin(ctx)
            if cos_sin is None:
                raise NotImplementedError(f"{self.name}: the position encoding must offer its cos/sin table")
        # convolved queries have rows of their own: the tokens behind still need the projected ones
        q_rows = rows[:, : self.q_cols]
        if self.taps is not None:
            q_rows = torch.empty((tokens, self.q_cols), dtype=rows.dtype, device=rows.device)
        planes = len(cache.planes) == 2                        # [pages, kv heads, page, dim] each
        keys, values = (cache.k, cache.v) if planes else (cache.planes[0], None)
        K.attention_prepare(rows, q_rows, cos_sin, ctx, table, (keys, values) if planes else keys, q_heads=heads, k_heads=self.num_kv_heads,
                            dim=self.head_dim, value_width=self.v_cols, taps=self.taps,
                            state=cache.state if self.conv_taps > 1 else None, state_offset=self.state_offset,
                            q_weight=self.q_norm_weight, k_weight=self.k_norm_weight, eps=self.eps, write=cache.owner)
        num_pages, _, page, width = keys.shape
        if planes and K.paged_attention_takes_sinks(rows.dtype, self.head_dim, page) and out.stride(0) % 8 == 0:
            o = K.paged_attention(q_rows, keys, values, table, ctx, heads, self.num_kv_heads, self.head_dim, self.scale, None,
                                  sink=self.sink, softcap=self.softcap, out=None if self.has_gate else out)
            o = o.unflatten(1, (heads, self.value_dim))
        else:
            if planes:
                key_strides = value_strides = (self.num_kv_heads * page * width, page * width, width)
            else:
                values = keys.view(-1)[self.k_cols:]
                key_strides = (page * width, self.head_dim, width)
                value_strides = (page * width, self.value_dim, width)
            direct = out.unflatten(1, (heads, self.value_dim))
            o = K.attention_dims(
                q_rows.unflatten(1, (heads, self.head_dim)), keys, values, table, ctx, value_heads=self.num_kv_heads,
                group=heads // self.num_kv_heads, maps=1, key_width=self.head_dim, value_width=self.value_dim,
                page_size=page, num_pages=num_pages, key_strides=key_strides, value_strides=value_strides,
                scale=self.scale, sink=self.sink, softcap=self.softcap, out=None if self.has_gate else direct)
        if self.has_gate:
            gate = rows[:, self.g_col:self.g_col + self.out_cols]
            if out.is_contiguous():
                K.sigmoid_gate_mul(o, gate, out=out)
            else:                                  # columns of a shared output matrix
                out.copy_(K.sigmoid_gate_mul(o, gate))


MIXERS.register("grouped_attention", GroupedAttention)

__all__ = ["GroupedAttention"]
