"""Zokepel: a decoder-only design whose layers run a sequence mixer and a clamped gated feed-forward IN PARALLEL on the same
fp32 residual stream, each behind its own weighted RMS norm:

    x <- x + mixer(w1 x / rms(x)) + ff(w2 x / rms(x))                rms(x) = sqrt(mean(x^2) + eps)

The stream starts as ``scale * embed[token]`` plus a sinusoidal position vector; the output is ``head . (w_final x / rms(x))``.
A contiguous range of layers may be LOOPED: layers ``start .. stop-1`` run ``times`` times in a row with the same weights, every
pass with a cache and states of its own, and the embedding output joins the stream again right before every pass but the
first.  A "layer run" below is one execution of one layer.  Three kinds of mixers (``models/mixers.py``):

* ``delta``: gated delta rule, one decay per head, silu output gate;
* ``channel_delta``: gated delta rule, one decay per head and key row (low-rank), sigmoid output gate (low-rank);
* ``parallel``: two branches on one input, each RMS-normed over the width before half their sum is taken — softmax attention
  with unit-RMS queries and keys, a query temperature by position and a learned bias per logarithmic distance bucket (left),
  and RWKV-style time mixing with a bonus for the current token (right).

The feed-forward is ``Wdown (g sigmoid(1.702 g) (u + 1))`` on the clamped gate and up projections; a layer may have none.  The
layer list, every size and every constant come from the checkpoint's ``config.json``:

    {"architecture": "Zokepel", "width", "vocab", "norm": {"eps"}, "embedding": {"scale"}, "loop": {"start", "stop", "times"}?,
     "layers": [{"type": "delta" | "channel_delta", "mixer": {"heads", "kv_heads", "dim", "vdim", "conv"}, "mlp": ...},
                {"type": "parallel", "mixer": {"left": {"heads", "kv_heads", "dim", "vdim", "scale", "bias_max",
                                                        "q_temp": {"coef", "every"}?},
                                               "right": {"heads", "dim"}}, "mlp": ...}]}
    mlp: null | {"kind": "dense", "ff", "limit"}

The ranks of the low-rank projections and the rows of the distance-bias tables are the extents of the checkpoint's tensors.
Checkpoint tensors: ``embed``, ``head``, ``final.norm``, ``l<i>.norm1|norm2``, ``l<i>.mix.*`` (see the mixers' ``load``),
``l<i>.mlp.{gate,up,down}``; linear weights are [out, in].  The model runs ragged paged batches only (``forward_ragged``); the
serving engine owns the caches, the state slots and their reuse.

Reference: none — the reference serves whatever HF returns (reference llmctl/serve/server.py:127-160)."""
from __future__ import annotations

from dataclasses import dataclass, field
from pathlib import Path
from typing import Any, Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from ..ops import dual_norm as dnops
from ..ops import elementwise as eops
from ..ops import functional as ops
from .ffn import GatedClampedMLP
from .mixers import (BonusMemory, BonusMemorySpec, BranchPair, DeltaRule, DeltaRuleSpec, SoftcapWindowAttention,
                     SoftcapWindowAttentionSpec)
from .registry import Architecture, register_architecture

MIXER_TYPES = ("delta", "channel_delta", "parallel")
GATE_ALPHA = 1.702              # the feed-forward's gate is g * sigmoid(1.702 g)
POSITION_BASE = 10000.0         # base of the sinusoidal position vector


@dataclass
class BranchPairSpec:
    left: SoftcapWindowAttentionSpec
    right: BonusMemorySpec


@dataclass
class ZokepelLayer:
    type: str
    mixer: Any                              # the mixer's spec
    ff: int                                 # inner size of the feed-forward, 0 = none
    limit: float = 0.0


@dataclass
class ZokepelConfig:
    name: str = "zokepel"
    width: int = 256
    vocab_size: int = 512
    norm_eps: float = 1e-6
    embed_scale: float = 1.0
    loop: Optional[Tuple[int, int, int]] = None          # (start, stop, times)
    layers: List[ZokepelLayer] = field(default_factory=list)
    max_position_embeddings: int = 1 << 20               # positions are computed: bounded by the cache pool only
    raw: Dict[str, Any] = field(default_factory=dict)

    @classmethod
    def from_dict(cls, d: Dict[str, Any], name: str = "zokepel") -> "ZokepelConfig":
        layers: List[ZokepelLayer] = []
        for i, l in enumerate(d["layers"]):
            m = l["mixer"]
            if l["type"] in ("delta", "channel_delta"):
                ch = l["type"] == "channel_delta"
                heads = int(m["heads"])
                spec: Any = DeltaRuleSpec(heads=heads, kv_heads=int(m.get("kv_heads", heads)), dim=int(m["dim"]),
                                          vdim=int(m.get("vdim", m["dim"])), conv=int(m["conv"]), per_channel=ch,
                                          decay_rank=int(m.get("decay_rank", 0)) if ch else 0,
                                          gate_rank=int(m.get("gate_rank", 0)) if ch else 0,
                                          gate_act="sigmoid" if ch else "silu")
                pairs = [(spec.heads, spec.kv_heads)]
            elif l["type"] == "parallel":
                a, r = m["left"], m["right"]
                t = a.get("q_temp")
                heads = int(a["heads"])
                left = SoftcapWindowAttentionSpec(heads=heads, kv_heads=int(a.get("kv_heads", heads)), dim=int(a["dim"]),
                                                  vdim=int(a.get("vdim", a["dim"])), scale=float(a["scale"]), distance_bias=False,
                                                  sink_one=False, value_norm=False, bias=False, out_gate=False, qk_norm=True,
                                                  q_temp=(float(t["coef"]), float(t["every"])) if t else None,
                                                  bias_rows=int(a.get("bias_rows", 0)), bias_max=float(a["bias_max"]))
                spec = BranchPairSpec(left, BonusMemorySpec(heads=int(r["heads"]), dim=int(r["dim"]), decay_rank=int(r.get("decay_rank", 0))))
                pairs = [(left.heads, left.kv_heads)]
            else:
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r} (known: {MIXER_TYPES})")
            if any(h % g for h, g in pairs):
                raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
            mlp = l.get("mlp")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            layers.append(ZokepelLayer(l["type"], spec, int(mlp["ff"]), float(mlp["limit"])) if mlp is not None
                          else ZokepelLayer(l["type"], spec, 0))
        loop = None
        lp = d.get("loop")
        if lp and int(lp["stop"]) > int(lp["start"]):
            loop = (int(lp["start"]), int(lp["stop"]), int(lp.get("times", 1)))
            if not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1:
                raise ValueError(f"loop {lp} does not fit {len(layers)} layers")
        return cls(name=name, width=int(d["width"]), vocab_size=int(d["vocab"]), norm_eps=float((d.get("norm") or {}).get("eps", 1e-6)),
                   embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)), loop=loop, layers=layers, raw=d)

    def to_dict(self) -> Dict[str, Any]:
        return dict(self.raw)

    def runs(self) -> List[Tuple[int, bool]]:
        """The layer runs in order: (layer index, whether the embedding output joins the stream before it)."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, False) for i in range(n)]
        start, stop, times = self.loop
        out: List[Tuple[int, bool]] = [(i, False) for i in range(start)]
        for t in range(times):
            out += [(i, t > 0 and i == start) for i in range(start, stop)]
        return out + [(i, False) for i in range(stop, n)]

    def num_parameters(self) -> int:
        with torch.device("meta"):
            m = ZokepelModel(self, dtype=torch.bfloat16, device="meta")
        return sum(p.numel() for p in m.parameters())


class ZokepelBlock(nn.Module):
    def __init__(self, cfg: ZokepelConfig, layer: ZokepelLayer, dtype, device):
        super().__init__()
        W = cfg.width
        self.norm_w = nn.ParameterList([nn.Parameter(torch.ones(W, dtype=torch.float32, device=device)) for _ in range(2 if layer.ff else 1)])
        if layer.type == "parallel":
            self.mixer: nn.Module = BranchPair(W, SoftcapWindowAttention(W, layer.mixer.left, cfg.norm_eps, dtype, device),
                                               BonusMemory(W, layer.mixer.right, cfg.norm_eps, dtype, device), device)
        else:
            self.mixer = DeltaRule(W, layer.mixer, cfg.norm_eps, dtype, device)
        self.mlp = GatedClampedMLP(W, layer.ff, layer.limit, GATE_ALPHA, dtype, device) if layer.ff else None


class ZokepelModel(nn.Module):
    ragged = True           # runs ragged paged batches through ``forward_ragged`` (serve/engine.py)
    stateful = True         # keeps per-sequence states: the engine hands out state slots with the pages

    def __init__(self, cfg: ZokepelConfig, *, dtype=torch.bfloat16, device=None):
        super().__init__()
        self.cfg, self.dtype = cfg, dtype
        self.embed = nn.Parameter(torch.empty(cfg.vocab_size, cfg.width, dtype=dtype, device=device))
        self.blocks = nn.ModuleList([ZokepelBlock(cfg, l, dtype, device) for l in cfg.layers])
        self.final_w = nn.Parameter(torch.ones(cfg.width, dtype=torch.float32, device=device))
        self.head = nn.Parameter(torch.empty(cfg.vocab_size, cfg.width, dtype=dtype, device=device))
        self.register_buffer("pos_freq", dnops.sinusoid_frequencies(cfg.width, POSITION_BASE).to(device), persistent=False)
        self.runs = cfg.runs()

    # ---- weights ---------------------------------------------------------------------------------------
    def load_state(self, tensors: Dict[str, torch.Tensor]) -> None:
        """``tensors``: checkpoint names -> tensors (any float type; converted to the model's)."""
        dev = self.embed.device

        def get(name: str) -> torch.Tensor:
            if name not in tensors:
                raise KeyError(f"checkpoint has no tensor {name!r}")
            return tensors[name].to(dev)
        with torch.no_grad():
            self.embed.copy_(get("embed"))
            self.head.copy_(get("head"))
            self.final_w.copy_(get("final.norm").float())
            for i, blk in enumerate(self.blocks):
                for s in range(len(blk.norm_w)):
                    blk.norm_w[s].copy_(get(f"l{i}.norm{s + 1}").float())
                blk.mixer.load(get, f"l{i}.mix.")
                if blk.mlp is not None:
                    blk.mlp.load(get, f"l{i}.mlp.")

    def init_random(self, seed: int = 0) -> None:
        g = torch.Generator().manual_seed(seed)
        with torch.no_grad():
            for name, p in self.named_parameters():
                leaf = name.rsplit(".", 1)[-1]
                if leaf == "speed":
                    p.copy_(torch.exp(torch.rand(p.shape, generator=g) * 2.0 - 1.5))
                elif leaf == "dt_bias":
                    p.copy_(torch.rand(p.shape, generator=g) * 4.0 - 5.0)
                elif leaf == "w_0":
                    p.copy_(torch.rand(p.shape, generator=g) * 6.0 - 6.0)
                elif leaf == "mu":
                    p.copy_(torch.rand(p.shape, generator=g))
                elif leaf in ("u", "rel"):
                    p.copy_(0.5 * torch.randn(p.shape, generator=g))
                elif leaf == "conv_w":
                    p.copy_(torch.randn(p.shape, generator=g) / p.shape[-1] ** 0.5)
                elif p.dim() == 1:
                    p.copy_((1.0 + 0.1 * torch.randn(p.shape, generator=g)).to(p.dtype))
                else:
                    p.copy_((torch.randn(p.shape, generator=g) / p.shape[-1] ** 0.5).to(p.dtype))
        for m in self.modules():
            if isinstance(m, SoftcapWindowAttention):
                m._table = None

    # ---- caches and states -----------------------------------------------------------------------------
    def cache_bytes_per_block(self, block_size: int) -> int:
        it = torch.empty((), dtype=self.dtype).element_size()
        return sum(self.cfg.layers[li].mixer.left.cache_width for li, _ in self.runs if self.cfg.layers[li].type == "parallel") * block_size * it

    def allocate_caches(self, num_blocks: int, block_size: int, device, state_slots: int = 1) -> List[Any]:
        """One entry per layer run: the tuple of fp32 state tensors ``[state_slots, ...]`` of a delta-rule run; of a parallel run
        ``(paged [pages, block_size, G (d + e)] key/value cache, the right branch's state tensors)``."""
        def own(mixer: nn.Module) -> Any:
            if isinstance(mixer, BranchPair):
                return own(mixer.left), own(mixer.right)
            if mixer.stateful:
                return tuple(torch.zeros(state_slots, *shape, dtype=torch.float32, device=device) for shape in mixer.state_shapes())
            return torch.zeros(mixer.cache_shape(num_blocks, block_size), dtype=self.dtype, device=device)
        return [own(self.blocks[li].mixer) for li, _ in self.runs]

    # ---- forward ---------------------------------------------------------------------------------------
    @torch.no_grad()
    def forward_ragged(self, batch, caches: List[Any], layer_trace: Optional[list] = None) -> torch.Tensor:
        """``batch``: serve.ragged.RaggedBatch.  Returns fp32 logits [len(batch.out_rows), vocab]."""
        cfg, dt, eps, runs = self.cfg, self.dtype, self.cfg.norm_eps, self.runs
        x, x0 = dnops.embed_sinusoid(batch.tokens, batch.positions, self.embed, cfg.embed_scale, self.pos_freq,
                                     want_copy=any(rejoin for _, rejoin in runs))

        def norms(r: int):
            return list(self.blocks[runs[r][0]].norm_w) if r < len(runs) else []
        hs = dnops.residual_dual_norm(None, None, x, eps, norms(0), dt) if runs else []
        for r, (li, _) in enumerate(runs):
            blk = self.blocks[li]
            m = blk.mixer(hs[0], batch, caches[r])
            f = blk.mlp(hs[1]) if blk.mlp is not None else None
            # residual update, the embedding output where the next pass begins and the next layer's norms in one pass over the rows
            add = x0 if r + 1 < len(runs) and runs[r + 1][1] else None
            if layer_trace is None:
                hs = dnops.residual_dual_norm(m, f, x, eps, norms(r + 1), dt, add=add)
            else:
                dnops.residual_dual_norm(m, f, x, eps, [], dt)
                layer_trace.append(x.clone())
                hs = dnops.residual_dual_norm(None, None, x, eps, norms(r + 1), dt, add=add)
        if batch.num_out == 0:                  # a step that only fills the caches and states
            return torch.empty(0, cfg.vocab_size, dtype=torch.float32, device=x.device)
        y = eops.rmsnorm_rows(x, batch.out_rows, self.final_w, eps, dt)
        if y.is_cuda and dt == torch.bfloat16:
            if ops.kernel_config().gemm == "native" and ops._gemm_ok(y, self.head) and self.head.shape[0] % 8 == 0:
                return ops.gemm_raw(y, self.head, out_dtype=torch.float32)
            return torch.mm(y, self.head.t(), out_dtype=torch.float32)
        return torch.nn.functional.linear(y.float(), self.head.float())


def _complete_config(cfg: ZokepelConfig, directory) -> None:
    """Sizes that ``config.json`` leaves to the checkpoint: the ranks of the low-rank projections and the rows of the
    distance-bias tables are extents of its tensors."""
    from safetensors import safe_open
    with safe_open(str(Path(directory) / "model.safetensors"), framework="pt") as f:
        def rows(name: str) -> int:
            return int(f.get_slice(name).get_shape()[0])
        for i, l in enumerate(cfg.layers):
            p = f"l{i}.mix."
            if l.type == "channel_delta":
                l.mixer.decay_rank = l.mixer.decay_rank or rows(p + "a1")
                l.mixer.gate_rank = l.mixer.gate_rank or rows(p + "g1")
            elif l.type == "parallel":
                l.mixer.left.bias_rows = l.mixer.left.bias_rows or rows(p + "left.rel")
                l.mixer.right.decay_rank = l.mixer.right.decay_rank or rows(p + "right.w1")


def _load_weights(model: ZokepelModel, directory) -> None:
    from safetensors.torch import load_file
    model.load_state(load_file(str(Path(directory) / "model.safetensors")))


def build_zokepel(cfg: ZokepelConfig, *, dtype=torch.bfloat16, device=None, seed: int = 42, **_ignored) -> ZokepelModel:
    m = ZokepelModel(cfg, dtype=dtype, device=device)
    m.init_random(seed)
    return m


register_architecture(Architecture(name="Zokepel", config_from_dict=ZokepelConfig.from_dict, config_type=ZokepelConfig,
                                   build=build_zokepel, load_weights=_load_weights, complete_config=_complete_config))


def example_config(width: int = 40, vocab: int = 72, pattern: str = "CDPC", ff: str = "1101", loop: Optional[Tuple[int, int, int]] = (1, 3, 2),
                   heads: int = 4, kv_heads: int = 2, dim: int = 6, vdim: int = 10, conv: int = 3, decay_rank: int = 5, gate_rank: int = 3,
                   att_heads: int = 4, att_kv_heads: int = 2, att_dim: int = 8, att_vdim: int = 12, att_scale: Optional[float] = None,
                   bias_rows: int = 8, bias_max: float = 30.0, q_temp: Optional[Tuple[float, float]] = (0.4, 7), mix_heads: int = 3,
                   mix_dim: int = 5, mix_rank: int = 4, ff_size: int = 24, limit: float = 1.5, scale: float = 3.0,
                   eps: float = 1e-5) -> Dict[str, Any]:
    """A small configuration dictionary for tests, benchmarks and examples.  ``pattern``: one character per layer for its
    mixer (D delta rule with a decay per head, C with a decay per key row, P attention beside time mixing); ``ff``: one
    character per layer, 1 = the layer has a feed-forward; ``loop`` = (start, stop, times) or None."""
    layers: List[Dict[str, Any]] = []
    for i, ch in enumerate(pattern):
        if ch == "P":
            left: Dict[str, Any] = {"heads": att_heads, "kv_heads": att_kv_heads, "dim": att_dim, "vdim": att_vdim,
                                    "scale": att_dim ** -0.5 if att_scale is None else att_scale, "bias_max": bias_max, "bias_rows": bias_rows}
            if q_temp:
                left["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
            layer: Dict[str, Any] = {"type": "parallel", "mixer": {"left": left, "right": {"heads": mix_heads, "dim": mix_dim, "decay_rank": mix_rank}}}
        else:
            mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}
            if ch == "C":
                mixer.update(decay_rank=decay_rank, gate_rank=gate_rank)
            layer = {"type": "channel_delta" if ch == "C" else "delta", "mixer": mixer}
        layer["mlp"] = {"kind": "dense", "ff": ff_size, "limit": limit} if ff[i % len(ff)] == "1" else None
        layers.append(layer)
    cfg: Dict[str, Any] = {"architecture": "Zokepel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale},
                           "layers": layers}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg
