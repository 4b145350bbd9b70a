"""Softmax attention with rotary positions over a ring of key / value rows, grouped key/value heads and an element-wise
sigmoid gate on the heads' outputs, with the variations models differ in as parameters of the spec:

    q, k <- [shortconv]( W h )                       a short causal filter per channel, its last inputs kept as state
    q, k <- rmsnorm_row(.) * w                       one norm over the WHOLE projection, before the heads are split, or
    q, k <- rmsnorm_head(.) * w                      one per head, with a weight of the head's size shared by all heads
    q    <- q * (1 + coef ln(floor((p + 1) / every) + 1))      at position p (query temperature)
    q, k <- rotate(., position)                      rotary.RotarySpec (partial dimensions, rescaled frequencies), in the "rotate
                                                     half" pairing or (``rot_layout`` "interleaved") neighbours 2i, 2i + 1
    v     = W_v h,  or the keys as they are before the rotation (``own_values`` False),  or, mixed with the values an
            earlier layer projected for the same token, (1 - lam) * W_v h + lam * v_first (lam learned; the mix is cached)
    s_h(i, j) = scale * q_h(i).k_g(j)  [- slope_h * (i - j)]  [-> cap * tanh(s / cap)],     slope_h = 2^(-8 (h + 1) / H)
    visible:    j <= i  [and i - j < window]  [and j // chunk == i // chunk]
    w = exp(s) / (sum_visible exp(s) [+ exp(sink_h)])         the sink is a number per head without key or value, learned or
                                                              (``fixed_sink``) a constant of the design
    out = W_o( concat_h( sum_j w v_g(j) ) * sigmoid(W_g h) )

With ``maps`` = 2 every head carries two score maps (differential attention): the q and k projections hold ``[map 0 | map 1]``
per head, both maps attend over the same values, and the head's output is

    o = a_0 - lam * a_1,   lam = exp(lq1 . lk1) - exp(lq2 . lk2) + diff,       o <- o / sqrt(mean(o^2) + eps) * (1 - diff)

(``lq1`` ... ``lk2`` learned vectors of the layer, ``diff`` a constant of the spec).  ``gate`` False: no sigmoid gate.

A layer with ``kv_from`` set has no key / value tensors: it appends nothing and reads the ring of the layer it names
(whose keys are stored after norm and rotation), with its own queries, mask, sink and gate.

The kernels turn pairs in the "rotate half" layout; a checkpoint with interleaved pairs has the rows of its query and key
projections (and what weighs them channel by channel) reordered once at load time, the same way on both sides of the dot
product.  ``project`` False: the layer keeps the input and output projections itself (stacked with others); ``in_rows`` hands
over the rows, ``attend`` is what remains.

Cache: ``[B, R, G * maps * dim]`` keys and ``[B, R, G * vdim]`` values, position j at slot ``j % R`` (csrc/rotary_attn.cu).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import List, Optional, Tuple

import torch
import torch.nn as nn
from torch.nn import functional as F

from . import _native as N
from .rotary import RotarySpec
from .short_conv import ShortConv


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass
class SoftmaxAttentionSpec:
    width: int
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    eps: float
    rotary: RotarySpec = field(default_factory=lambda: RotarySpec(0))
    softcap: float = 0.0                 # 0: scores are not capped
    window: Optional[int] = None         # sliding window (None: none)
    chunk: Optional[int] = None          # chunk-local mask (None: none)
    sink: bool = False
    qk_norm: bool = False
    conv_taps: int = 0                   # 0: no short convolution on q and k
    own_values: bool = True              # False: the values are the un-rotated keys
    kv_from: Optional[int] = None        # index of the layer whose ring this layer reads
    maps: int = 1                        # score maps per head; 2: the difference of two softmax maps with a unit norm per head
    diff: float = 0.0                    # the constant of the two-map combination
    gate: bool = True                    # sigmoid(W_g h) on the heads' outputs
    head_norm: bool = False              # a norm per head on q and k (qk_norm: over the whole projection)
    temp_coef: float = 0.0               # query temperature
    temp_every: int = 0                  # 0: none
    distance_bias: bool = False          # scores fall by slope_h per position of distance
    v_mix: bool = False                  # values are mixed with those of another layer (``attend``'s ``first_values``)
    rot_layout: str = "half"             # which dimensions turn together: "half" (i, i + dims/2) | "interleaved" (2i, 2i + 1)
    fixed_sink: Optional[float] = None   # a sink of this score on every head (``sink``: one learned per head)

    def __post_init__(self):
        if self.rot_layout not in ("half", "interleaved"):
            raise ValueError(f"rotary layout {self.rot_layout!r}")
        if self.rot_layout == "interleaved" and not self.own_values:
            raise ValueError("values taken from the keys keep the keys' order of dimensions")
        if self.sink and self.fixed_sink is not None:
            raise ValueError("a sink is either learned or a constant")
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} query heads over {self.kv_heads} key/value heads")
        if not self.own_values and self.vdim != self.dim:
            raise ValueError("values taken from the keys have the keys' size")
        if self.maps not in (1, 2):
            raise ValueError(f"{self.maps} score maps per head (1 or 2)")
        if self.maps > 1 and not self.own_values:
            raise ValueError("values taken from the keys need one score map per head")
        per_head = self.head_norm or self.temp_every > 0 or self.v_mix
        if per_head and (self.qk_norm or self.maps > 1 or not self.own_values or self.kv_from is not None):
            raise ValueError("a norm per head, a query temperature and mixed values go with one score map, keys and values of the "
                             "layer's own and no norm over the whole projection")
        if self.temp_every < 0:
            raise ValueError(f"a query temperature that steps every {self.temp_every} positions")
        if self.rotary.dims > self.dim:
            raise ValueError(f"{self.rotary.dims} rotated dimensions in heads of {self.dim}")

    def head_order(self) -> torch.Tensor:
        """Where every dimension of a stored query / key head sits in the checkpoint's."""
        order = list(range(self.dim))
        if self.rot_layout == "interleaved":
            half = self.rotary.dims // 2
            for i in range(half):
                order[i], order[i + half] = 2 * i, 2 * i + 1
        return torch.tensor(order, dtype=torch.long)

    @property
    def by_head(self) -> bool:
        """Whether q, k and v are prepared head by head (ll_qk_head_append)."""
        return self.head_norm or self.temp_every > 0 or self.v_mix

    @property
    def reach(self) -> Optional[int]:
        """A query at position i reads no key before ``i - reach + 1`` (None: unbounded)."""
        bounds = [b for b in (self.window, self.chunk) if b is not None]
        return min(bounds) if bounds else None


class SoftmaxAttention(nn.Module):
    def __init__(self, spec: SoftmaxAttentionSpec, dtype: torch.dtype, device, project: bool = True) -> None:
        super().__init__()
        s = self.spec = spec
        kw = dict(dtype=dtype, device=device)
        f32 = dict(dtype=torch.float32, device=device)
        hd, gd, gv, hv = s.heads * s.maps * s.dim, s.kv_heads * s.maps * s.dim, s.kv_heads * s.vdim, s.heads * s.vdim
        self.owner = s.kv_from is None
        names, at = [("q", hd)] + ([("k", gd)] if self.owner else []) + ([("v", gv)] if self.owner and s.own_values else []) \
            + ([("g", hv)] if s.gate else []), 0
        self.cols = {}
        for name, n in names:
            self.cols[name] = at
            at += n
        self.n_in = at
        self.w_in = nn.Parameter(torch.zeros((pad8(self.n_in), s.width), **kw), requires_grad=False) if project else None
        self.conv_channels = hd + (gd if self.owner else 0)
        self.conv = ShortConv(self.conv_channels, s.conv_taps, False, device) if s.conv_taps > 0 else None
        normed = s.qk_norm or s.head_norm
        self.q_norm = nn.Parameter(torch.ones(s.dim if s.head_norm else hd, **f32), requires_grad=False) if normed else None
        self.k_norm = nn.Parameter(torch.ones(s.dim if s.head_norm else gd, **f32), requires_grad=False) if normed and self.owner else None
        self.v_lambda = 0.0                            # lam of the value mix, read at load time
        self.register_buffer("slopes", torch.tensor([2.0 ** (-8.0 * (h + 1) / s.heads) for h in range(s.heads)],
                                                    dtype=torch.float64).to(**f32) if s.distance_bias else None, persistent=False)
        self.sink = nn.Parameter(torch.full((s.heads * s.maps,), s.fixed_sink or 0.0, **f32), requires_grad=False) \
            if s.sink or s.fixed_sink is not None else None
        self.register_buffer("freq", s.rotary.frequencies(device), persistent=False)
        self.diff_lambda = 0.0                         # lam of the two-map combination, formed at load time
        # queries that are neither filtered, normed nor turned are read where the input projection left them
        self.plain_q = self.conv is None and not s.qk_norm and s.rotary.dims == 0 and not s.by_head
        self.w_o = nn.Parameter(torch.zeros((s.width, hv), **kw), requires_grad=False) if project else None

    @property
    def out_cols(self) -> int:
        """What ``attend`` puts out per token."""
        return self.spec.heads * self.spec.vdim

    def state_shapes(self, B: int) -> List[Tuple[int, ...]]:
        return [self.conv.state_shape(B)] if self.conv is not None else []

    def cache_shapes(self, B: int, ring: int) -> List[Tuple[int, ...]]:
        s = self.spec
        return [(B, ring, s.kv_heads * s.maps * s.dim), (B, ring, s.kv_heads * s.vdim)] if self.owner else []

    def _stored(self, w: torch.Tensor) -> torch.Tensor:
        """Rows of q or k (whole heads of ``dim``) in the stored order of dimensions."""
        if self.spec.rot_layout == "half":
            return w
        heads = w.reshape(-1, self.spec.dim, *w.shape[1:])
        return heads[:, self.spec.head_order().to(w.device)].reshape(w.shape)

    def in_rows(self, get) -> torch.Tensor:
        """The rows of the stacked input projection, in the order of ``cols``."""
        return torch.cat([self._stored(get(n)) if n in "qk" else get(n) for n in self.cols], dim=0)

    def load(self, get) -> None:
        """``get(suffix)`` returns the tensor '<layer>.mix.<suffix>'."""
        s = self.spec
        if self.w_in is not None:
            self.w_in.zero_()
            self.w_in[: self.n_in].copy_(self.in_rows(get))
            self.w_o.copy_(get("o"))
        if self.conv is not None:
            self.conv.load(torch.cat([self._stored(get(n + ".conv").float()) for n in ("qk" if self.owner else "q")], dim=0))
        if self.q_norm is not None:
            self.q_norm.copy_(self._stored(get("q.norm").float()))
        if self.k_norm is not None:
            self.k_norm.copy_(self._stored(get("k.norm").float()))
        if s.sink:
            self.sink.copy_(get("sink").float())
        if s.maps == 2:
            l = [get(n).double() for n in ("lq1", "lk1", "lq2", "lk2")]
            self.diff_lambda = float(torch.exp((l[0] * l[1]).sum()) - torch.exp((l[2] * l[3]).sum()) + s.diff)
        if s.v_mix:
            self.v_lambda = float(get("vmix").float())

    def values(self, proj: torch.Tensor) -> torch.Tensor:
        """The columns of the input projection's output that hold this layer's own values."""
        s = self.spec
        return proj[:, self.cols["v"]: self.cols["v"] + s.kv_heads * s.vdim]

    def forward(self, u: torch.Tensor, B: int, T: int, pos_ids: torch.Tensor, caches, conv_state=None, splits: int = 1,
                form: int = 0) -> torch.Tensor:
        return F.linear(self.attend(F.linear(u, self.w_in), B, T, pos_ids, caches, conv_state, splits, form), self.w_o)

    def attend(self, proj: torch.Tensor, B: int, T: int, pos_ids: torch.Tensor, caches, conv_state=None, splits: int = 1,
               form: int = 0, first_values: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        """``proj``: the stacked input projection's output; ``caches`` = (keys, values) of this layer or of the one it reads;
        ``first_values``: the values mixed into this layer's (``v_mix``), of the same tokens; ``out``: a column slice to write to.
        Returns the gated heads ``[B*T, heads * vdim]`` (before the output projection)."""
        s = self.spec
        c = self.cols
        kc, vc = caches
        M = B * T
        dtc = N.dtype_code(proj.dtype)
        ring = kc.shape[1]
        st = N.stream()
        hd = s.heads * s.maps * s.dim
        if self.conv is not None:
            src = self.conv(proj, 0, conv_state, pos_ids, B, T, proj.dtype)
            q_at, k_at = N.ptr(src), N.ptr_at(src, hd)
        else:
            src = proj
            q_at, k_at = N.ptr_at(proj, c["q"]), (N.ptr_at(proj, c["k"]) if self.owner else None)
        v_at = N.ptr_at(proj, c["v"]) if "v" in c else None
        if self.plain_q:
            q, q_ptr, q_stride = None, q_at, src.stride(0)
        else:
            q = torch.empty((M, hd), dtype=proj.dtype, device=proj.device)
            q_ptr, q_stride = N.ptr(q), hd
        if s.by_head:
            if s.v_mix and (first_values is None or first_values.shape != (M, s.kv_heads * s.vdim)):
                raise ValueError("a layer with mixed values needs the other layer's values of the same tokens")
            first = first_values if s.v_mix else None
            N.call("ll_qk_head_append", q_at, src.stride(0), k_at, src.stride(0), v_at, proj.stride(0), N.ptr(first),
                   first.stride(0) if first is not None else 0, float(self.v_lambda), dtc,
                   N.ptr(self.q_norm), N.ptr(self.k_norm), float(s.eps), N.ptr(self.freq), s.rotary.dims, float(s.temp_coef),
                   s.temp_every, N.ptr(pos_ids), N.ptr(q), N.ptr(kc), N.ptr(vc), B, T, s.heads, s.kv_heads, s.dim, s.vdim, ring, st)
        elif self.owner or not self.plain_q:
            N.call("ll_qk_rotary_append_maps", None if self.plain_q else q_at, src.stride(0), k_at if self.owner else None, src.stride(0),
                   v_at, proj.stride(0), dtc, N.ptr(self.q_norm), N.ptr(self.k_norm), float(s.eps), N.ptr(self.freq), s.rotary.dims,
                   N.ptr(pos_ids), N.ptr(q), N.ptr(kc), N.ptr(vc), B, T, s.heads, s.kv_heads, s.dim, s.vdim, ring, s.maps, st)
        if s.distance_bias and s.maps > 1:
            form = 1                                   # two biased maps have no tensor-core form
        gate_at, gate_stride = (N.ptr_at(proj, c["g"]), proj.stride(0)) if s.gate else (None, 0)
        scratch = None
        if splits > 1 or (s.maps > 1 and (form != 0 or not N.call_ret("ll_softmax_attn_tensor_form", dtc, T, s.dim, s.vdim, q_stride,
                                                                       gate_stride, splits))):
            scratch = torch.empty(N.call_ret("ll_softmax_attn_scratch_bytes", M, s.heads * s.maps, s.vdim, splits) // 4,
                                  dtype=torch.float32, device=proj.device)
        y = out if out is not None else torch.empty((M, s.heads * s.vdim), dtype=proj.dtype, device=proj.device)
        N.call("ll_softmax_attn_rows", q_ptr, q_stride, gate_at, gate_stride, N.ptr(kc), N.ptr(vc), dtc, N.ptr(pos_ids),
               N.ptr(self.sink), N.ptr(self.slopes), float(s.scale), float(s.softcap), B, T, s.heads, s.kv_heads, s.dim, s.vdim,
               s.window or 0, s.chunk or 0, ring, splits, form, s.maps, float(self.diff_lambda), float(1.0 - s.diff), float(s.eps), N.ptr(scratch), N.ptr(y),
               y.stride(0), st)
        return y
