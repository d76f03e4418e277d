"""Grouped-query attention whose queries and keys are normed, with the mechanisms that go with it.

With ``H`` query heads and ``G`` key/value heads (query head h reads key/value head ``h // (H / G)``), query/key heads of
``head_dim`` entries and value heads of ``v_head_dim``:

    q, k, v = Wq x, Wk x, Wv x          (+ biases with ``qkv_bias``)
    ``qk_norm="head"``   every query and key head u becomes u / sqrt(mean(u^2) + eps) * w, one weight for all query heads and one
                         for all key heads
    ``qk_norm="row"``    the same over a token's whole query row and its whole key row, weights of that size
    ``position``         then q and k turn by position (a ``rope_span`` at the start of the head; None: nothing turns)
    ``heat=(c, every)``  then q is multiplied by 1 + c ln(floor((p + 1) / every) + 1) at position p
    ``value_mix``        ``"mix"``: v <- (1 - l) v + l v_first, v_first the values of the same token in the layer built with
                         ``"first"``, which comes earlier in the run order; the mixed v is what the cache keeps.  Either layer
                         loads the number l (the first one does not use it)
    score(p, j) = (q . k_j) * scale  [+ rel[bucket(p - j), h] with ``bias_rows``]       softmax over the keys in sight
    ``window``           the last ``window`` keys;  ``chunk``: the keys of the query's own chunk of that many positions, chunks
                         counted from position 0;  neither: every key up to the query's own
    ``gate``             the concatenated heads are multiplied entry by entry by sigmoid(Wg x)
    out = Wo heads       (+ a bias with ``out_bias``)

``bucket(n)`` with R = ``bias_rows`` rows, half of them (h = R // 2) for single distances: n itself below h; from there on
``h + floor((R - h) log_b(n / h))`` with ``b = bias_max / h``, never beyond R - 1: from ``bias_max`` on every distance shares the last row.  The table is laid out by distance once, when it is
bound, so that the attention kernels look a distance up.

Norms, turn, temperature and mixing happen in one kernel on the float32 value of each projected entry, and what attention
reads is rounded once (``ops.qk_norm_append``)."""
from __future__ import annotations

import math
from typing import Dict, List, Mapping, Optional

import torch

from .. import ops
from ..cache.manager import CallCacheView, PagedKVNeed
from ..config.spec import PartSpec
from ..weights.loader import TensorSpec
from .base import Mixer, StepContext, build_part, register_mixer
from .linear_recurrence import _stack_padded
from .mlp import _stack

FIRST_VALUES = ("first_values",)         # where the "first" layer of a step leaves its values (``StepContext.step_cache``)


def distance_bucket(n: int, rows: int, farthest: float) -> int:
    half = rows // 2
    if n < half:
        return n
    share = math.log(n / half) / math.log(farthest / half)
    # a distance that lies on a bucket's edge belongs to the bucket it opens, whichever way the logarithms round
    return min(rows - 1, half + math.floor(share * (rows - half) + 1e-12 * rows))


def distance_buckets(rows: int, farthest: float) -> List[int]:
    """The bucket of every distance from 0 up to the first one from which all share the last bucket."""
    return [distance_bucket(n, rows, farthest) for n in range(max(math.ceil(farthest), rows // 2) + 1)]


@register_mixer("normed_attention")
class NormedAttentionMixer(Mixer):
    capture_safe = True

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, v_head_dim: Optional[int] = None,
                 qk_norm: Optional[str] = "head", eps: float = 1e-6, position: Optional[PartSpec] = None, scale: Optional[float] = None,
                 window: Optional[int] = None, chunk: Optional[int] = None, qkv_bias: bool = False, out_bias: bool = False,
                 gate: bool = False, heat: Optional[tuple] = None, value_mix: Optional[str] = None, bias_rows: Optional[int] = None,
                 bias_max: Optional[float] = None, names: Optional[Mapping[str, str]] = None):
        v_head_dim = head_dim if v_head_dim is None else v_head_dim
        if min(hidden_size, num_heads, num_kv_heads, head_dim, v_head_dim) <= 0:
            raise ValueError("normed_attention: every size must be positive")
        if num_heads % num_kv_heads:
            raise ValueError(f"normed_attention: {num_heads} query heads cannot share {num_kv_heads} key/value heads")
        if qk_norm not in (None, "head", "row"):
            raise ValueError(f"normed_attention: qk_norm={qk_norm!r} is not 'head', 'row' or None")
        if value_mix not in (None, "first", "mix"):
            raise ValueError(f"normed_attention: value_mix={value_mix!r} is not 'first', 'mix' or None")
        if (window is not None and chunk is not None) or (window or 1) <= 0 or (chunk or 1) <= 0:
            raise ValueError(f"normed_attention: window={window} or chunk={chunk} must be positive, and only one of them given")
        if heat is not None and not heat[1] > 0.0:
            raise ValueError(f"normed_attention: the temperature's step {heat[1]} must be positive")
        if bias_rows is not None and (bias_rows < 2 or bias_max is None or not bias_max > bias_rows // 2):
            raise ValueError(f"normed_attention: {bias_rows} rows of distances need at least 2 and a farthest distance beyond half of them, "
                             f"got {bias_max}")
        self.hidden_size, self.num_heads, self.num_kv_heads = int(hidden_size), int(num_heads), int(num_kv_heads)
        self.head_dim, self.v_head_dim = int(head_dim), int(v_head_dim)
        # rows of the cache and heads of the query: wide enough for keys and values alike
        self.row_dim = (max(self.head_dim, self.v_head_dim) + 7) // 8 * 8
        if self.row_dim > 1024:
            raise ValueError(f"normed_attention: head sizes {head_dim} and {v_head_dim} are not supported; rows of at most 1024 entries")
        self.qk_norm, self.eps = qk_norm, float(eps)
        self.scale = float(scale) if scale is not None else 1.0 / math.sqrt(float(head_dim))
        if bias_rows is not None and not self.scale > 0.0:
            raise ValueError(f"normed_attention: a bias by distance needs a positive scale, got {self.scale}")
        self.window = int(window) if window is not None else None
        self.chunk = int(chunk) if chunk is not None else None
        self.qkv_bias, self.out_bias, self.gate = bool(qkv_bias), bool(out_bias), bool(gate)
        self.heat = (float(heat[0]), float(heat[1])) if heat is not None else None
        self.value_mix = value_mix
        self.bias_rows = int(bias_rows) if bias_rows is not None else None
        self.bias_max = float(bias_max) if bias_max is not None else None
        self.position = build_part("position", position) if position is not None else None
        if self.position is not None and (not hasattr(self.position, "dims") or getattr(self.position, "offset", 0)
                                          or self.position.head_dim != self.head_dim or self.position.unit_rms_eps is not None):
            raise ValueError("normed_attention: the position rule is a 'rope_span' at the start of this layer's heads, without unit heads")
        self.names = {"q": "q", "k": "k", "v": "v", "o": "o", "g": "g", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b", "o_bias": "o.b",
                      "q_norm": "q.norm", "k_norm": "k.norm", "rel": "rel", "lambda": "vmix"}
        self.names.update(names or {})
        self.q_dim, self.kv_dim, self.v_dim = self.num_heads * self.head_dim, self.num_kv_heads * self.head_dim, self.num_kv_heads * self.v_head_dim
        self.w_in = self.b_in = self.w_o = self.b_o = self.q_weight = self.k_weight = self.bias = None
        self.lam = 0.0
        self._gate_at = 0

    def cache_need(self):
        return PagedKVNeed(self.num_kv_heads, self.row_dim, self.window, chunk=self.chunk)

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        nm, h = self.names, self.hidden_size
        heads_out = self.num_heads * self.v_head_dim
        specs = {nm["q"]: TensorSpec((self.q_dim, h)), nm["k"]: TensorSpec((self.kv_dim, h)), nm["v"]: TensorSpec((self.v_dim, h)),
                 nm["o"]: TensorSpec((h, heads_out))}
        if self.qkv_bias:
            specs.update({nm["q_bias"]: TensorSpec((self.q_dim,)), nm["k_bias"]: TensorSpec((self.kv_dim,)), nm["v_bias"]: TensorSpec((self.v_dim,))})
        if self.out_bias:
            specs[nm["o_bias"]] = TensorSpec((h,))
        if self.gate:
            specs[nm["g"]] = TensorSpec((heads_out, h))
        if self.qk_norm is not None:
            one = ("one_plus_normal", 0.01)
            row = self.qk_norm == "row"
            specs[nm["q_norm"]] = TensorSpec((self.q_dim if row else self.head_dim,), init=one)
            specs[nm["k_norm"]] = TensorSpec((self.kv_dim if row else self.head_dim,), init=one)
        if self.value_mix is not None:
            specs[nm["lambda"]] = TensorSpec((), init=("normal", 0.3))
        if self.bias_rows is not None:
            specs[nm["rel"]] = TensorSpec((self.bias_rows, self.num_heads), init=("normal", 0.5))
        return specs

    def _wide_rows(self, t: torch.Tensor) -> torch.Tensor:
        """Rows of ``v_head_dim`` per head, each head padded with zero rows to ``row_dim``: the attention's output has that many
        entries per head, zero past the value's own."""
        if self.row_dim == self.v_head_dim:
            return t
        out = t.new_zeros((self.num_heads, self.row_dim) + tuple(t.shape[1:]))
        out[:, :self.v_head_dim] = t.view((self.num_heads, self.v_head_dim) + tuple(t.shape[1:]))
        return out.view((self.num_heads * self.row_dim,) + tuple(t.shape[1:]))

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        nm = self.names
        qkv = _stack([tensors[nm[r]] for r in ("q", "k", "v")])
        self.b_in = _stack([tensors[nm[r + "_bias"]] for r in ("q", "k", "v")]) if self.qkv_bias else None
        if self.gate:
            self.w_in, offsets = _stack_padded([qkv, self._wide_rows(tensors[nm["g"]])])        # one product makes q | k | v | the gate's input
            self._gate_at = offsets[1]
        else:
            self.w_in = qkv
        if self.b_in is not None:
            bias = self.b_in.new_zeros(self.w_in.shape[0])
            bias[:self.b_in.shape[0]] = self.b_in
            self.b_in = bias
            if self.b_in.dtype != self.w_in.dtype:             # one product, one operand type: float32 wins
                self.w_in, self.b_in = self.w_in.float(), self.b_in.float()
        self.w_o = self._wide_rows(tensors[nm["o"]].t().contiguous()).t().contiguous()
        self.b_o = tensors[nm["o_bias"]].contiguous() if self.out_bias else None
        if self.qk_norm is not None:                            # norms are float32
            self.q_weight, self.k_weight = tensors[nm["q_norm"]].float().contiguous(), tensors[nm["k_norm"]].float().contiguous()
        if self.value_mix is not None:
            self.lam = float(tensors[nm["lambda"]].float().cpu())                              # read once, at load
        if self.bias_rows is not None:
            rel = tensors[nm["rel"]].float()
            at = torch.tensor(distance_buckets(self.bias_rows, self.bias_max), dtype=torch.long, device=rel.device)
            self.bias = rel[at].t().contiguous()                                               # [heads, distances]

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: CallCacheView, owns_cache: bool) -> torch.Tensor:
        out = ctx.empty(x.shape[0], self.hidden_size)
        ops.linear(self._attend(x, ctx, cache, owns_cache), self.w_o, self.b_o, out)
        return out

    def forward_for_residual(self, x: torch.Tensor, ctx: StepContext, cache: CallCacheView, owns_cache: bool) -> torch.Tensor:
        return ops.linear_for_residual(self._attend(x, ctx, cache, owns_cache), self.w_o, self.b_o)

    def _attend(self, x: torch.Tensor, ctx: StepContext, cache: CallCacheView, owns_cache: bool) -> torch.Tensor:
        """Everything up to the output projection: ``[tokens, heads * row_dim]``."""
        if cache.kind != "paged" or not owns_cache:
            raise RuntimeError("normed_attention needs a paged key/value cache of its own")
        n = x.shape[0]
        proj = ctx.empty(n, self.w_in.shape[0])
        ops.linear(x, self.w_in, self.b_in, proj)
        first = None
        if self.value_mix is not None:
            at = self.q_dim + self.kv_dim
            if self.value_mix == "first":
                ctx.step_cache[FIRST_VALUES] = proj[:, at:at + self.v_dim]
            else:
                first = ctx.step_cache.get(FIRST_VALUES)
                if first is None:
                    raise RuntimeError("normed_attention: no earlier layer of this step has left its values to be mixed in")
        q = ctx.empty(n, self.num_heads, self.row_dim)
        pos = self.position
        dims = pos.dims if pos is not None else 0
        ops.qk_norm_append(proj, q, ctx.positions, cache, ctx.tables[cache.group], ctx.tok_seg, self.num_heads, self.num_kv_heads, self.head_dim,
                           self.v_head_dim, self.row_dim, norm=self.qk_norm, qw=self.q_weight, kw=self.k_weight, eps=self.eps,
                           inv_freq=pos.table(x.device) if dims else None, mag=pos.magnitude if pos is not None else 1.0, rot_dims=dims,
                           interleaved=pos.interleaved if pos is not None else False, heat=self.heat, v_first=first, lam=self.lam)
        attn = ctx.empty(n, self.num_heads * self.row_dim)
        ops.attention(q, cache, attn, ctx, self.num_heads, self.num_kv_heads, self.row_dim, self.window, self.scale, chunk=self.chunk,
                      bias=self.bias)
        if self.gate:
            ops.sigmoid_mul(attn, proj[:, self._gate_at:self._gate_at + attn.shape[1]])
        return attn
