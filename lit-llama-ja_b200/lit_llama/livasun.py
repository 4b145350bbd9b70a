"""Livasun: a decoder-only model of pre-norm sublayers on an fp32 stream that starts as ``embed[token] * s_e``,

    x <- x + mixer(ln1(x));      x <- x + ff(ln2(x))     (ff may be absent),      ln(x) = (x - mean) / sqrt(var + eps) * w + b

with mixers of three kinds in whatever order ``config.json`` lists them:

* ``mamba2``    - selective state space with one decay per head and token (recurrence.StateSpaceMixer);
* ``lightning`` - linear attention with a constant decay per head (recurrence.ConstantDecayAttention);
* ``attention`` - softmax attention over a sliding window (softmax_attention.SoftmaxAttention) without rotation: a norm per
  head on q and k, a query temperature that grows with the position, a bias linear in the distance, and values mixed with
  those the model's first such layer projected for the same token.

Feed-forward: silu-gated, or a mixture of squared-relu experts (moe.MoE) with sigmoid scores, a correction for the choice,
groups scored by their two best experts, and an always-on expert.  Logits: ``head . ln_f(x)``.

Per-sequence memory: the inputs of the state-space layers' short convolutions, the states of both recurrences, one key ring
and one value ring per attention layer (the values as mixed).  stepping.RingStateDecoder holds it; its step function is the
package's common one.
"""
from __future__ import annotations

import json
from dataclasses import dataclass, field
from pathlib import Path
from typing import Dict, List, Optional, Tuple, Union

import torch
import torch.nn as nn
from torch.nn import functional as F

from . import _native as N
from .feed_forward import DenseFF
from .moe import MoE, MoESpec
from .recurrence import ConstantDecayAttention, ConstantDecaySpec, StateSpaceMixer, StateSpaceSpec, pad8
from .rotary import RotarySpec
from .softmax_attention import SoftmaxAttention, SoftmaxAttentionSpec
from .stepping import RingStateDecoder, add_layer_norm, head_logits

ARCHITECTURE = "Livasun"


@dataclass
class LivasunLayer:
    kind: str                                          # "mamba2" | "lightning" | "attention"
    mixer: Union[StateSpaceSpec, ConstantDecaySpec, SoftmaxAttentionSpec]
    mlp: Union[None, int, MoESpec]                     # None: no feed-forward; a number: dense of that inner size


@dataclass
class LivasunConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    layers: List[LivasunLayer] = field(default_factory=list)
    values_of: Optional[int] = None                    # the layer whose values the layers with mixed values take in

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def n_layer(self) -> int:
        return len(self.layers)

    @property
    def block_size(self) -> int:
        """No position table: any length the memory is sized for."""
        return 1 << 30

    @classmethod
    def from_dict(cls, cfg: dict, shapes: Optional[Dict[str, Tuple[int, ...]]] = None) -> "LivasunConfig":
        """From the dictionary of a ``config.json``; sizes it leaves out are taken from the tensors' shapes."""
        shapes = shapes or {}

        def pick(value, name, axis, div=1):
            if value is not None:
                return int(value)
            if name in shapes:
                return shapes[name][axis] // div
            raise KeyError(f"config.json gives no size that tensor {name!r} would determine, and the tensor is absent")

        width = pick(cfg.get("width"), "embed", 1)
        vocab = pick(cfg.get("vocab"), "embed", 0)
        eps = float(cfg["norm"]["eps"])
        layers: List[LivasunLayer] = []
        any_mixed = False                  # the first attention layer that asks for mixed values only gives its own to the others
        for i, lc in enumerate(cfg["layers"]):
            kind, m, p = lc.get("type"), lc["mixer"], f"l{i}.mix."
            if kind == "mamba2":
                heads = pick(m.get("heads"), p + "A_log", 0)
                mixer = StateSpaceSpec(width=width, heads=heads, vdim=pick(m.get("vdim"), p + "o", 1, heads), state=int(m["state"]),
                                       groups=int(m.get("groups", 1)), norm_groups=int(m.get("norm_groups", 1)),
                                       taps=pick(m.get("conv"), p + "conv", 1), eps=eps)
            elif kind == "lightning":
                decay = [float(d) for d in m["decay"]]
                heads = int(m["heads"]) if m.get("heads") is not None else len(decay)
                mixer = ConstantDecaySpec(width=width, heads=heads, dim=pick(m.get("dim"), p + "q", 0, heads),
                                          vdim=pick(m.get("vdim"), p + "v", 0, heads), decay=decay, eps=eps)
            elif kind == "attention":
                dim = pick(m.get("dim"), p + "q.norm", 0)
                heads, kv_heads = pick(m.get("heads"), p + "q", 0, dim), pick(m.get("kv_heads"), p + "k", 0, dim)
                mask, temp = m.get("mask") or {}, m.get("q_temp") or {}
                mixer = SoftmaxAttentionSpec(
                    width=width, heads=heads, kv_heads=kv_heads, dim=dim, vdim=pick(m.get("vdim"), p + "v", 0, kv_heads),
                    scale=float(m["scale"]) if m.get("scale") is not None else dim ** -0.5, eps=eps, rotary=RotarySpec(0),
                    window=int(mask["size"]) if mask.get("size") is not None else None, gate=False, head_norm=True,
                    temp_coef=float(temp.get("coef", 0.0)), temp_every=int(temp.get("every", 0)), distance_bias=True,
                    v_mix=bool(m.get("v_mix", False)) and any_mixed)
                any_mixed = any_mixed or bool(m.get("v_mix", False))
            else:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            layers.append(LivasunLayer(kind, mixer, cls._mlp(lc.get("mlp"), i, width, pick)))
        mixed = [i for i, lc in enumerate(cfg["layers"]) if lc.get("type") == "attention" and lc["mixer"].get("v_mix")]
        if len({layers[i].mixer.kv_heads * layers[i].mixer.vdim for i in mixed}) > 1:
            raise ValueError(f"layers {mixed} mix their values but have value projections of different sizes")
        return cls(vocab=vocab, width=width, eps=eps, embed_scale=float((cfg.get("embedding") or {}).get("scale", 1.0)), layers=layers,
                   values_of=mixed[0] if len(mixed) > 1 else None)

    @staticmethod
    def _mlp(f: Optional[dict], i: int, width: int, pick) -> Union[None, int, MoESpec]:
        q = f"l{i}.mlp."
        if f is None:
            return None
        if f.get("kind", "dense") == "dense":
            return pick(f.get("ff"), q + "up", 0)
        if f["kind"] == "moe":
            r = f["router"]
            g = r.get("groups") or {}
            count = int(g.get("count", 1))
            shared = f.get("shared")
            return MoESpec(width=width, experts=pick(r.get("experts"), q + "router", 0), top=int(r["top"]),
                           ff=pick((f.get("expert") or {}).get("ff"), q + "e0.up", 0), limit=float("inf"),
                           shared_ff=pick(shared.get("ff"), q + "shared.up", 0) if shared is not None else None, shared_gate=False,
                           router_bias=False, score="sigmoid", groups=count, keep_groups=int(g.get("keep", count)), group_top=2,
                           correction=True, weight_scale=float(r.get("scale", 1.0)), unit="relu2")
        raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")


class LayerNormWeights(nn.Module):
    def __init__(self, width: int, device) -> None:
        super().__init__()
        f32 = dict(dtype=torch.float32, device=device)
        self.w = nn.Parameter(torch.ones(width, **f32), requires_grad=False)
        self.b = nn.Parameter(torch.zeros(width, **f32), requires_grad=False)

    def load(self, get, name: str) -> None:
        self.w.copy_(get(name).float())
        self.b.copy_(get(name + ".b").float())


_MIXERS = {"mamba2": StateSpaceMixer, "lightning": ConstantDecayAttention, "attention": SoftmaxAttention}


class LivasunBlock(nn.Module):
    def __init__(self, index: int, layer: LivasunLayer, cfg: LivasunConfig, dtype, device) -> None:
        super().__init__()
        self.index, self.kind = index, layer.kind
        self.norm1 = LayerNormWeights(cfg.width, device)
        self.mix = _MIXERS[layer.kind](layer.mixer, dtype, device)
        self.mlp = None
        if isinstance(layer.mlp, MoESpec):
            self.mlp = MoE(layer.mlp, dtype, device)
        elif layer.mlp is not None:
            self.mlp = DenseFF(cfg.width, layer.mlp, "silu_glu", dtype, device)
        self.norm2 = LayerNormWeights(cfg.width, device) if self.mlp is not None else None
        self.n_states = len(self.mix.state_shapes(1))

    def load(self, get) -> None:
        p = f"l{self.index}."
        self.norm1.load(get, p + "norm1")
        self.mix.load(lambda s: get(p + "mix." + s))
        if self.mlp is not None:
            self.norm2.load(get, p + "norm2")
            self.mlp.load(lambda s: get(p + "mlp." + s))


class Livasun(RingStateDecoder):
    architecture = ARCHITECTURE

    def __init__(self, config: LivasunConfig, dtype: torch.dtype = torch.bfloat16, device="cuda") -> None:
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("Livasun runs in bfloat16 or float32")
        self.config = config
        self.dtype, self.device = dtype, torch.device(device)
        kw = dict(dtype=dtype, device=self.device)
        self.embed = nn.Parameter(torch.empty((config.vocab, config.width), **kw), requires_grad=False)
        self.blocks = nn.ModuleList(LivasunBlock(i, l, config, dtype, self.device) for i, l in enumerate(config.layers))
        self.final_norm = LayerNormWeights(config.width, self.device)
        self.head = nn.Parameter(torch.zeros((pad8(config.vocab), config.width), **kw), requires_grad=False)
        self._attn = [b.mix for b in self.blocks if b.kind == "attention"]      # one ring each, in order

    # ------------------------------------------------------------------ weights
    @torch.no_grad()
    def load_tensors(self, get) -> None:
        """``get(name)`` returns the checkpoint tensor of that name (any float dtype, CPU or GPU)."""
        self.embed.copy_(get("embed"))
        self.head.zero_()
        self.head[: self.config.vocab].copy_(get("head"))
        self.final_norm.load(get, "final.norm")
        for b in self.blocks:
            b.load(get)

    @classmethod
    def from_dir(cls, path, dtype: torch.dtype = torch.bfloat16, device="cuda") -> "Livasun":
        """A folder with ``config.json`` and ``model.safetensors``."""
        from .safetensors_io import SafetensorsFile

        path = Path(path)
        with open(path / "config.json") as f:
            cfg = json.load(f)
        with SafetensorsFile(path / "model.safetensors") as st:
            model = cls(LivasunConfig.from_dict(cfg, st.shapes()), dtype=dtype, device=device)
            model.load_tensors(st.get)
        return model.eval()

    # ------------------------------------------------------------------ memory
    def _ring_reaches(self) -> List[Optional[int]]:
        return [a.spec.reach for a in self._attn]

    def _ring_shapes(self, n: int, B: int, ring: int) -> List[Tuple[int, ...]]:
        return self._attn[n].cache_shapes(B, ring)

    def _state_shapes(self, B: int) -> List[Tuple[int, ...]]:
        return [s for b in self.blocks for s in b.mix.state_shapes(B)]

    # ------------------------------------------------------------------ forward
    def _forward_portion(self, idx: torch.Tensor, pos_ids: torch.Tensor, sel) -> torch.Tensor:
        cfg = self.config
        B, T = idx.shape
        M, E = B * T, cfg.width
        dev = idx.device
        act = N.dtype_code(self.dtype)
        x = torch.empty((M, E), dtype=torch.float32, device=dev)
        N.call("ll_embed_scaled", N.ptr(self.embed), act, N.ptr(idx.reshape(-1).contiguous()), float(cfg.embed_scale), N.ptr(x), None, act,
               M, E, N.stream())
        sms = N.call_ret("ll_sm_count")
        pending = None                     # the sublayer result that is not in the stream yet
        first_values = None                # what layer `values_of` projected for this pass's tokens
        si = ci = 0
        for i, blk in enumerate(self.blocks):
            h = torch.empty((M, E), dtype=self.dtype, device=dev)
            add_layer_norm(x, pending, 1.0, blk.norm1.w, blk.norm1.b, cfg.eps, h, self.dtype)
            if self.layer_probe is not None and i > 0:
                self.layer_probe(i - 1, x)
            if blk.kind == "attention":
                spec, ring = blk.mix.spec, self._rings[ci]
                span = min(spec.reach if spec.reach is not None else (1 << 30), ring)
                # few queries: share the look-back among blocks, down to 32 keys each
                splits = max(1, min(64, (2 * sms) // max(1, (M * spec.heads + 3) // 4), (span + 31) // 32))
                proj = F.linear(h, blk.mix.w_in)
                y = blk.mix.attend(proj, B, T, pos_ids, self.kv_caches[2 * ci:2 * ci + 2], None, splits, first_values=first_values)
                if i == cfg.values_of:
                    first_values = blk.mix.values(proj)
                pending = F.linear(y, blk.mix.w_o)
                ci += 1
            else:
                pending = blk.mix(h, B, T, pos_ids, self.states[si:si + blk.n_states])
                si += blk.n_states
            if blk.mlp is not None:
                h2 = torch.empty((M, E), dtype=self.dtype, device=dev)
                add_layer_norm(x, pending, 1.0, blk.norm2.w, blk.norm2.b, cfg.eps, h2, self.dtype)
                pending = blk.mlp(h2)
        if sel is not None and len(sel) == 0:      # the step only fills the memory
            return torch.empty((B, 0, cfg.vocab), dtype=torch.float32, device=dev)
        add_layer_norm(x, pending, 1.0, None, None, cfg.eps, None, self.dtype)
        if self.layer_probe is not None:
            self.layer_probe(cfg.n_layer - 1, x)
        if sel is not None:
            ridx = (torch.arange(B, device=dev)[:, None] * T + torch.tensor(sel, device=dev, dtype=torch.long)[None]).reshape(-1)
            x = x.index_select(0, ridx).contiguous()
        xn = torch.empty((x.shape[0], E), dtype=self.dtype, device=dev)
        add_layer_norm(x, None, 1.0, self.final_norm.w, self.final_norm.b, cfg.eps, xn, self.dtype)
        return head_logits(xn, self.head, cfg.vocab).reshape(B, -1, cfg.vocab)
