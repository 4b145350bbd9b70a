"""Zekonex: a decoder-only model of parallel layers on an fp32 stream that starts as ``embed[token] * s_e``; a layer has one norm,
and both of its sublayers read its output:

    h = rmsnorm(x) * w;      x <- x + r * ( mixer(h) + ff(h) )          (ff may be absent)

with mixers of three kinds in whatever order ``config.json`` lists them:

* ``attention``        - softmax attention (softmax_attention.SoftmaxAttention), causal over the whole past, the first dimensions
  of every query and key head turned in neighbouring pairs, a constant sink of score 0 in the softmax denominator;
* ``delta``            - gated delta rule (recurrence.GatedDeltaMixer);
* ``latent_attention`` - latent attention (latent_attention.LatentAttention) without a gate, causal over the whole past.

Feed-forward: the clamped gated unit with biases (feed_forward.ClampedUnit).  Logits: ``head . (rmsnorm(x) * w_f)``.

A range of layers may run several times in a row with the same weights (``loop``): every pass has rings and state of its own, and
right before its first layer a learned vector per pass joins the stream.  ``layer_runs`` lists what runs in order.

Both sublayers read one input and add to one stream, so a layer is two GEMMs around the mixer's kernels: [mixer; gate; up] stacked
into one input projection, [W_o | W_down] side by side into one output projection over rows [mixer's heads | unit], which the
mixer's last kernel and the unit write in place.  The bias of W_down, the multiplier r, the pass's vector and the next norm are one
launch.

Per-sequence memory, per run of a layer: a key and a value ring (attention), a ring of latent rows (latent attention), or the short
convolution's inputs and the memory (delta); stepping.RingStateDecoder holds it, its step function is the package's common one.
"""
from __future__ import annotations

import json
from dataclasses import dataclass, field
from pathlib import Path
from typing import Dict, List, NamedTuple, Optional, Tuple, Union

import torch
import torch.nn as nn
from torch.nn import functional as F

from . import _native as N
from .feed_forward import ClampedUnit
from .latent_attention import LatentAttention, LatentAttentionSpec
from .recurrence import GatedDeltaMixer, GatedDeltaSpec, pad8
from .rotary import RotarySpec
from .softmax_attention import SoftmaxAttention, SoftmaxAttentionSpec
from .stepping import RingStateDecoder, add_rms_norm, head_logits

ARCHITECTURE = "Zekonex"


@dataclass
class ZekonexLayer:
    kind: str                                          # "attention" | "delta" | "latent_attention"
    mixer: Union[SoftmaxAttentionSpec, GatedDeltaSpec, LatentAttentionSpec]
    ff: Optional[int]                                  # inner size of the feed-forward; None: the layer has none
    limit: float = float("inf")


@dataclass
class ZekonexLoop:
    start: int
    stop: int                                          # layers start .. stop - 1
    times: int


@dataclass
class ZekonexConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    embed_scale: float
    layers: List[ZekonexLayer] = field(default_factory=list)
    loop: Optional[ZekonexLoop] = None

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def n_layer(self) -> int:
        return len(self.layers)

    @property
    def block_size(self) -> int:
        """No position table bounds the length: any the memory is sized for."""
        return 1 << 30

    def layer_runs(self) -> List[Tuple[int, Optional[int]]]:
        """(layer, the pass it opens or None) in the order they run."""
        n, lp = self.n_layer, self.loop
        if lp is None:
            return [(i, None) for i in range(n)]
        return ([(i, None) for i in range(lp.start)]
                + [(i, t if i == lp.start else None) for t in range(lp.times) for i in range(lp.start, lp.stop)]
                + [(i, None) for i in range(lp.stop, n)])

    @classmethod
    def from_dict(cls, cfg: dict, shapes: Optional[Dict[str, Tuple[int, ...]]] = None) -> "ZekonexConfig":
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
        layers: List[ZekonexLayer] = []
        for i, lc in enumerate(cfg["layers"]):
            kind, m, p = lc.get("type"), lc["mixer"], f"l{i}.mix."
            if kind == "attention":
                dim = int(m["dim"])
                kv_heads = pick(m.get("kv_heads"), p + "k", 0, dim)
                mixer = SoftmaxAttentionSpec(
                    width=width, heads=pick(m.get("heads"), p + "q", 0, dim), kv_heads=kv_heads, dim=dim,
                    vdim=pick(m.get("vdim"), p + "v", 0, kv_heads), scale=float(m["scale"]) if m.get("scale") is not None else dim ** -0.5,
                    eps=eps, rotary=RotarySpec.from_dict(m.get("rot"), dim), gate=False, rot_layout="interleaved", fixed_sink=0.0)
            elif kind == "delta":
                heads = pick(m.get("heads"), p + "A_log", 0)
                kv_heads = int(m["kv_heads"]) if m.get("kv_heads") is not None else heads
                mixer = GatedDeltaSpec(width=width, heads=heads, kv_heads=kv_heads, dim=pick(m.get("dim"), p + "q", 0, kv_heads),
                                       vdim=pick(m.get("vdim"), p + "norm", 0), taps=pick(m.get("conv"), p + "q.conv", 1), eps=eps)
            elif kind == "latent_attention":
                dim, rot_dim = int(m["dim"]), int(m.get("rot_dim") or 0)
                heads = pick(m.get("heads"), p + "uk", 0, dim)
                rotary = RotarySpec.from_dict(m.get("rot"), rot_dim) if rot_dim else RotarySpec(0)
                mixer = LatentAttentionSpec(
                    width=width, heads=heads, nope_dim=dim, rot_dim=rot_dim, v_dim=pick(m.get("vdim"), p + "uv", 0, heads),
                    kv_rank=pick(m.get("kv_rank"), p + "uk", 1), window=None,
                    scale=float(m["scale"]) if m.get("scale") is not None else (dim + rot_dim) ** -0.5, eps=eps, gate="none",
                    rot_layout="interleaved", rotary=rotary, exact_weights=True)
            else:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            f = lc.get("mlp")
            if f is None:
                layers.append(ZekonexLayer(kind, mixer, None))
            elif f.get("kind", "dense") == "dense":
                limit = float(f["limit"]) if f.get("limit") is not None else float("inf")
                layers.append(ZekonexLayer(kind, mixer, pick(f.get("ff"), f"l{i}.mlp.up", 0), limit))
            else:
                raise ValueError(f"layer {i}: unknown feed-forward kind {f.get('kind')!r}")
        loop = None
        if cfg.get("loop") is not None:
            lp = cfg["loop"]
            loop = ZekonexLoop(int(lp["start"]), int(lp["stop"]), pick(lp.get("times"), "loop.step", 0))
            if not (0 <= loop.start < loop.stop <= len(layers)) or loop.times < 1:
                raise ValueError(f"loop over layers {loop.start} .. {loop.stop - 1} of {len(layers)}, {loop.times} times")
        return cls(vocab=vocab, width=width, eps=eps, residual_mult=float(cfg.get("residual_mult", 1.0)),
                   embed_scale=float((cfg.get("embedding") or {}).get("scale", 1.0)), layers=layers, loop=loop)


_MIXERS = {"attention": SoftmaxAttention, "delta": GatedDeltaMixer, "latent_attention": LatentAttention}


class ZekonexBlock(nn.Module):
    def __init__(self, index: int, layer: ZekonexLayer, cfg: ZekonexConfig, dtype, device) -> None:
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        self.index, self.kind = index, layer.kind
        self.norm1 = nn.Parameter(torch.ones(cfg.width, dtype=torch.float32, device=device), requires_grad=False)
        self.mix = _MIXERS[layer.kind](layer.mixer, dtype, device, project=False)
        self.mlp = ClampedUnit(cfg.width, layer.ff, layer.limit, device) if layer.ff is not None else None
        ff = layer.ff or 0
        # where the unit's columns begin in the stacked projections; every part starts on a multiple of 8
        self.ff_in, self.ff_out = pad8(self.mix.n_in), pad8(self.mix.out_cols)
        self.n_out = pad8(self.ff_out + ff) if ff else self.mix.out_cols
        self.gaps = bool(ff) and (self.ff_out != self.mix.out_cols or self.n_out != self.ff_out + ff)
        self.w_in = nn.Parameter(torch.zeros((pad8(self.ff_in + 2 * ff), cfg.width), **kw), requires_grad=False)      # [mixer; gate; up]
        self.w_out = nn.Parameter(torch.zeros((cfg.width, self.n_out), **kw), requires_grad=False)                    # [W_o | W_down]

    def load(self, get) -> None:
        p = f"l{self.index}."
        self.norm1.copy_(get(p + "norm1").float())
        mix = (lambda s: get(p + "mix." + s))
        self.mix.load(mix)
        self.w_in.zero_()
        self.w_out.zero_()
        self.w_in[: self.mix.n_in].copy_(self.mix.in_rows(mix))
        self.w_out[:, : self.mix.out_cols].copy_(mix("o"))
        if self.mlp is not None:
            mlp = (lambda s: get(p + "mlp." + s))
            self.mlp.load(mlp)
            self.w_in[self.ff_in: self.ff_in + 2 * self.mlp.ff].copy_(self.mlp.in_rows(mlp))
            self.w_out[:, self.ff_out: self.ff_out + self.mlp.ff].copy_(self.mlp.down(mlp))


class LayerRun(NamedTuple):
    """One run of a layer: its memory is its own, whatever weights it shares with another run."""
    block: ZekonexBlock
    step: Optional[int]      # the pass it opens
    ring: int                # its ring among ``_rings``; -1: none
    cache_at: int            # its first tensor in ``kv_caches``
    state_at: int            # its first tensor in ``states``


class Zekonex(RingStateDecoder):
    architecture = ARCHITECTURE

    def __init__(self, config: ZekonexConfig, dtype: torch.dtype = torch.bfloat16, device="cuda") -> None:
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("Zekonex runs in bfloat16 or float32")
        self.config = config
        self.dtype, self.device = dtype, torch.device(device)
        kw = dict(dtype=dtype, device=self.device)
        f32 = dict(dtype=torch.float32, device=self.device)
        self.embed = nn.Parameter(torch.empty((config.vocab, config.width), **kw), requires_grad=False)
        self.blocks = nn.ModuleList(ZekonexBlock(i, l, config, dtype, self.device) for i, l in enumerate(config.layers))
        self.loop_step = nn.Parameter(torch.zeros((config.loop.times, config.width), **f32), requires_grad=False) if config.loop else None
        self.final_norm = nn.Parameter(torch.ones(config.width, **f32), requires_grad=False)
        self.head = nn.Parameter(torch.zeros((pad8(config.vocab), config.width), **kw), requires_grad=False)
        self.runs: List[LayerRun] = []
        rings = caches = states = 0
        for i, step in config.layer_runs():
            mix = self.blocks[i].mix
            n_caches, n_states = len(mix.cache_shapes(1, 1)), len(mix.state_shapes(1))
            self.runs.append(LayerRun(self.blocks[i], step, rings if n_caches else -1, caches, states))
            rings, caches, states = rings + (1 if n_caches else 0), caches + n_caches, states + n_states
        self._ringed = [r for r in self.runs if r.ring >= 0]

    # ------------------------------------------------------------------ weights
    @torch.no_grad()
    def load_tensors(self, get) -> None:
        """``get(name)`` returns the checkpoint tensor of that name (any float dtype, CPU or GPU)."""
        self.embed.copy_(get("embed"))
        self.head.zero_()
        self.head[: self.config.vocab].copy_(get("head"))
        self.final_norm.copy_(get("final.norm").float())
        if self.loop_step is not None:
            self.loop_step.copy_(get("loop.step").float())
        for b in self.blocks:
            b.load(get)

    @classmethod
    def from_dir(cls, path, dtype: torch.dtype = torch.bfloat16, device="cuda") -> "Zekonex":
        """A folder with ``config.json`` and ``model.safetensors``."""
        from .safetensors_io import SafetensorsFile

        path = Path(path)
        with open(path / "config.json") as f:
            cfg = json.load(f)
        with SafetensorsFile(path / "model.safetensors") as st:
            model = cls(ZekonexConfig.from_dict(cfg, st.shapes()), dtype=dtype, device=device)
            model.load_tensors(st.get)
        return model.eval()

    # ------------------------------------------------------------------ memory
    def _rotary_specs(self) -> List[RotarySpec]:
        return [b.mix.spec.rotary for b in self.blocks if b.kind == "latent_attention"]

    def _ring_reaches(self) -> List[Optional[int]]:
        return [None for _ in self._ringed]                                    # both attentions see the whole past

    def _ring_shapes(self, n: int, B: int, ring: int) -> List[Tuple[int, ...]]:
        return self._ringed[n].block.mix.cache_shapes(B, ring)

    def _state_shapes(self, B: int) -> List[Tuple[int, ...]]:
        return [s for r in self.runs for s in r.block.mix.state_shapes(B)]

    # ------------------------------------------------------------------ forward
    def _mixer(self, run: LayerRun, proj: torch.Tensor, B: int, T: int, pos_ids: torch.Tensor, sms: int, out: torch.Tensor) -> None:
        mix = run.block.mix
        spec = mix.spec
        M = B * T
        if run.block.kind == "delta":
            mix.mix(proj, B, T, pos_ids, self.states[run.state_at:run.state_at + 2], out)
        elif run.block.kind == "attention":
            # few queries: share the look-back among blocks, down to 32 keys each
            splits = max(1, min(64, (2 * sms) // max(1, (M * spec.heads + 3) // 4), (self._rings[run.ring] + 31) // 32))
            mix.attend(proj, B, T, pos_ids, self.kv_caches[run.cache_at:run.cache_at + 2], None, splits, out=out)
        else:
            splits = max(1, min(16, (2 * sms) // max(1, M * ((spec.heads + 31) // 32)), (self._rings[run.ring] + 63) // 64))
            mix.attend(proj, B, T, pos_ids, self.rope_table(spec.rotary), self.kv_caches[run.cache_at], splits, out=out)

    def _forward_portion(self, idx: torch.Tensor, pos_ids: torch.Tensor, sel) -> torch.Tensor:
        cfg = self.config
        B, T = idx.shape
        M, E = B * T, cfg.width
        dev = idx.device
        act = N.dtype_code(self.dtype)
        r = cfg.residual_mult
        x = torch.empty((M, E), dtype=torch.float32, device=dev)
        N.call("ll_embed_scaled", N.ptr(self.embed), act, N.ptr(idx.reshape(-1).contiguous()), float(cfg.embed_scale), N.ptr(x), None, act,
               M, E, N.stream())
        sms = N.call_ret("ll_sm_count")
        pending = bias = None              # the layer result that is not in the stream yet, the bias that goes with it
        for n, run in enumerate(self.runs):
            blk = run.block
            if self.layer_probe is not None and n > 0:     # the stream as the layer before left it, without the next pass's vector
                add_rms_norm(x, pending, r, bias, None, None, cfg.eps, None, self.dtype)
                self.layer_probe(n - 1, x)
                pending = bias = None
            h = torch.empty((M, E), dtype=self.dtype, device=dev)
            step = self.loop_step[run.step] if run.step is not None else None
            add_rms_norm(x, pending, r, bias, step, blk.norm1, cfg.eps, h, self.dtype)
            proj = F.linear(h, blk.w_in)
            rows = (torch.zeros if blk.gaps else torch.empty)((M, blk.n_out), dtype=self.dtype, device=dev)
            self._mixer(run, proj, B, T, pos_ids, sms, rows[:, : blk.mix.out_cols])
            bias = None
            if blk.mlp is not None:
                blk.mlp(proj[:, blk.ff_in:], rows[:, blk.ff_out: blk.ff_out + blk.mlp.ff])
                bias = blk.mlp.bias_down
            pending = F.linear(rows, blk.w_out)
        if sel is not None and len(sel) == 0 and self.layer_probe is None:      # the step only fills the memory
            return torch.empty((B, 0, cfg.vocab), dtype=torch.float32, device=dev)
        if sel is None and self.layer_probe is None:       # every row is asked for: the last sum and the final norm are one launch
            xn = torch.empty((M, E), dtype=self.dtype, device=dev)
            add_rms_norm(x, pending, r, bias, None, self.final_norm, cfg.eps, xn, self.dtype)
            return head_logits(xn, self.head, cfg.vocab).reshape(B, -1, cfg.vocab)
        add_rms_norm(x, pending, r, bias, None, None, cfg.eps, None, self.dtype)
        if self.layer_probe is not None:
            self.layer_probe(len(self.runs) - 1, x)
        if sel is not None:
            ridx = (torch.arange(B, device=dev)[:, None] * T + torch.tensor(sel, device=dev, dtype=torch.long)[None]).reshape(-1)
            x = x.index_select(0, ridx).contiguous()
        xn = torch.empty((x.shape[0], E), dtype=self.dtype, device=dev)
        add_rms_norm(x, None, 1.0, None, None, self.final_norm, cfg.eps, xn, self.dtype)
        return head_logits(xn, self.head, cfg.vocab).reshape(B, -1, cfg.vocab)
