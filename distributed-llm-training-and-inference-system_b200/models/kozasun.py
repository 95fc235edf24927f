"""Kozasun: a decoder-only design whose pre-normed sublayers (a sequence mixer, then a feed-forward) are joined by
hyper-connections: several parallel fp32 residual streams instead of one.  For every sublayer, with learned stream weights a, b
and M (indexed [from, to]):

    u = sum_s a_s x_s;   y = f(layernorm(u) w + bias);   x_t <- sum_s M[s, t] x_s + b_t y

The streams start as copies of ``scale * embed[token]``; the output is ``head . layernorm(sum_s x_s)``.  Three kinds of mixers
(``models/mixers.py``):

* ``attention``: grouped-query attention over chunks counted from position 0, with projection biases, an RMS norm over the whole
  q and k projections, rotation of halves and a learned sink per head;
* ``retention``: linear attention with a fixed decay per head on rotated queries and keys, heads at unit RMS, silu gate;
* ``latent_attention``: attention without positions whose keys and values are linear images of a cached low-rank latent, over a
  sliding window, with a sigmoid gate per head.

The feed-forward is a gated GELU (tanh form) or a mixture of gated-SiLU experts (``models/ffn.py``): sigmoid scores; a learned
correction added for the choice only; only experts of the best groups (sum of a group's two best choice scores) can be chosen;
the chosen scores times a constant, not renormalised; a shared expert for every token.  A layer may have none, and a layer may
use another layer's weights with a cache or state of its own (``weights_of``).  The layer list, every size and every
constant come from the checkpoint's ``config.json``:

    {"architecture": "Kozasun", "width", "vocab", "norm": {"eps"}, "embedding": {"scale"}, "streams",
     "layers": [{"type": "attention", "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"}, "rot": {"base", "dims"}}, ...},
                {"type": "retention", "mixer": {"heads", "dim", "vdim", "decay": [...], "rot": {"base", "dims"}}, ...},
                {"type": "latent_attention", "mixer": {"heads", "dim", "vdim", "kv_rank", "scale", "mask": {"size"}}, ...}]}
    and in every layer "mlp": null | {"kind": "dense", "ff"} |
        {"kind": "moe", "router": {"experts", "top", "scale", "groups": {"count", "keep"}?}, "expert": {"ff"}, "shared": {"ff"}?},
    "weights_of": j?

Checkpoint tensors: ``embed``, ``head``, ``final.norm`` (+ ``.b``), ``l<i>.norm1|norm2`` (+ ``.b``), ``l<i>.hc1|hc2.{in,out,mix}``,
``l<i>.mix.*`` (see the mixers' ``load``), ``l<i>.mlp.{gate,up,down}`` or ``l<i>.mlp.{router,correction,e<k>.*,shared.*}``; linear
weights are [out, in].  The model runs ragged paged batches only (``forward_ragged``); the serving engine owns the caches, the
state slots and their reuse.

Reference: none — the reference serves whatever HF returns (reference llmctl/serve/server.py:127-160)."""
from __future__ import annotations

from dataclasses import dataclass, field
from pathlib import Path
from typing import Any, Dict, List, Optional

import torch
import torch.nn as nn

from ..ops import functional as ops
from ..ops import hyper_norm as hops
from .ffn import GatedExpertMoE, GatedGeluMLP
from .mixers import (LatentAttention, LatentAttentionSpec, Retention, RetentionSpec, SoftcapWindowAttention, SoftcapWindowAttentionSpec)
from .registry import Architecture, register_architecture

MIXER_TYPES = ("attention", "retention", "latent_attention")
GROUP_BEST = 2                  # a group of experts is worth the sum of this many of its choice scores


@dataclass
class KozasunLayer:
    type: str
    mixer: Any                          # the mixer's spec
    mlp: Optional[Dict[str, Any]]
    owner: int                          # layer whose weights this one uses (its own index: it has tensors)


def _mixer_spec(i: int, kind: str, m: Dict[str, Any]) -> Any:
    heads, dim = int(m["heads"]), int(m["dim"])
    vdim = int(m.get("vdim", dim))
    rot = m.get("rot") or {}
    rot_dims, rot_base = int(rot.get("dims", 0)), float(rot.get("base", 10000.0))
    size = int((m.get("mask") or {}).get("size", 0))
    if rot_dims % 2 or rot_dims > dim:
        raise ValueError(f"layer {i}: the rotated part must be an even number of at most dim numbers")
    if kind == "attention":
        kv = int(m.get("kv_heads", heads))
        if heads % kv:
            raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
        return SoftcapWindowAttentionSpec(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=float(m["scale"]), distance_bias=False, sink_one=False,
                                          value_norm=False, bias=True, out_bias=False, out_gate=False, chunk=size, sink=True, proj_norm=True,
                                          rot_dims=rot_dims, rot_base=rot_base)
    if kind == "retention":
        decay = tuple(float(g) for g in m["decay"])
        if len(decay) != heads:
            raise ValueError(f"layer {i}: one decay per head, got {len(decay)} for {heads} heads")
        return RetentionSpec(heads=heads, dim=dim, vdim=vdim, decay=decay, rot_dims=rot_dims, rot_base=rot_base)
    if kind == "latent_attention":
        return LatentAttentionSpec(heads=heads, dim=dim, rot_dim=0, vdim=vdim, kv_rank=int(m["kv_rank"]), q_rank=0, scale=float(m["scale"]),
                                   rot_base=10000.0, head_gate=True, window=size)
    raise ValueError(f"layer {i}: unknown mixer type {kind!r} (known: {MIXER_TYPES})")


@dataclass
class KozasunConfig:
    name: str = "kozasun"
    width: int = 256
    vocab_size: int = 512
    norm_eps: float = 1e-5
    embed_scale: float = 1.0
    streams: Optional[int] = None                        # None: one plain residual stream (no stream weights)
    layers: List[KozasunLayer] = field(default_factory=list)
    max_position_embeddings: int = 1 << 20               # positions are computed: bounded by the cache pool only
    raw: Dict[str, Any] = field(default_factory=dict)

    @classmethod
    def from_dict(cls, d: Dict[str, Any], name: str = "kozasun") -> "KozasunConfig":
        layers: List[KozasunLayer] = []
        n = len(d["layers"])
        for i, l in enumerate(d["layers"]):
            owner, hops_left = i, n
            while d["layers"][owner].get("weights_of") is not None:
                owner, hops_left = int(d["layers"][owner]["weights_of"]), hops_left - 1
                if not 0 <= owner < n or hops_left < 0:
                    raise ValueError(f"layer {i}: weights_of does not lead to a layer with weights")
            if d["layers"][owner]["type"] != l["type"]:
                raise ValueError(f"layer {i}: it cannot use the weights of layer {owner}, which has another type")
            own = d["layers"][owner]
            mlp = own.get("mlp")
            if mlp is not None and mlp.get("kind") not in ("dense", "moe"):
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            layers.append(KozasunLayer(l["type"], _mixer_spec(i, l["type"], own["mixer"]), mlp, owner))
        streams = d.get("streams")
        if streams is not None and not 1 <= int(streams) <= hops.MAX_STREAMS:
            raise ValueError(f"streams must be 1 .. {hops.MAX_STREAMS}, got {streams}")
        return cls(name=name, width=int(d["width"]), vocab_size=int(d["vocab"]), norm_eps=float((d.get("norm") or {}).get("eps", 1e-5)),
                   embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)), streams=None if streams is None else int(streams),
                   layers=layers, raw=d)

    def to_dict(self) -> Dict[str, Any]:
        return dict(self.raw)

    def num_parameters(self) -> int:
        with torch.device("meta"):
            m = KozasunModel(self, dtype=torch.bfloat16, device="meta")
        return sum(p.numel() for p in m.parameters())


class SublayerNorm(nn.Module):
    """What surrounds a sublayer: its layer norm and its stream weights (fixed ones without hyper-connections)."""

    def __init__(self, cfg: KozasunConfig, device, want_fp32: bool):
        super().__init__()
        f32 = dict(dtype=torch.float32, device=device)
        S = cfg.streams or 1
        self.learned = cfg.streams is not None
        self.w = nn.Parameter(torch.ones(cfg.width, **f32))
        self.bias = nn.Parameter(torch.zeros(cfg.width, **f32))
        self.hc_in = nn.Parameter(torch.ones(S, **f32), requires_grad=False)
        self.hc_out = nn.Parameter(torch.ones(S, **f32), requires_grad=False)
        self.hc_mix = nn.Parameter(torch.eye(S, **f32), requires_grad=False)
        self.nxt = hops.NextNorm(self.hc_in, self.w, self.bias, want_fp32)
        self.streams = hops.StreamWeights(self.hc_in, self.hc_out, self.hc_mix)

    def load(self, get, prefix: str, q: int) -> None:
        self.w.copy_(get(f"{prefix}norm{q}").float())
        self.bias.copy_(get(f"{prefix}norm{q}.b").float())
        if self.learned:
            self.hc_in.copy_(get(f"{prefix}hc{q}.in").float().reshape(-1))
            self.hc_out.copy_(get(f"{prefix}hc{q}.out").float().reshape(-1))
            self.hc_mix.copy_(get(f"{prefix}hc{q}.mix").float().reshape(self.hc_mix.shape))


class KozasunBlock(nn.Module):
    def __init__(self, cfg: KozasunConfig, layer: KozasunLayer, dtype, device):
        super().__init__()
        W = cfg.width
        mixer = {"attention": SoftcapWindowAttention, "retention": Retention, "latent_attention": LatentAttention}[layer.type]
        self.mixer: nn.Module = mixer(W, layer.mixer, cfg.norm_eps, dtype, device)
        self.norm1 = SublayerNorm(cfg, device, want_fp32=False)
        mlp = layer.mlp
        self.mlp: Optional[nn.Module] = None
        if mlp is None:
            return
        self.norm2 = SublayerNorm(cfg, device, want_fp32=mlp["kind"] == "moe")
        if mlp["kind"] == "dense":
            self.mlp = GatedGeluMLP(W, int(mlp["ff"]), dtype, device)
        else:
            r, shared, groups = mlp["router"], mlp.get("shared"), mlp["router"].get("groups")
            self.mlp = GatedExpertMoE(W, int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"]), int(shared["ff"]) if shared else None, dtype,
                                      device, scale_input=False, softmax_scores=False, renormalise=False, shared_gate=False, correction=True,
                                      groups=(int(groups["count"]), int(groups["keep"])) if groups else None, group_best=GROUP_BEST,
                                      weight_scale=float(r.get("scale", 1.0)))


class KozasunModel(nn.Module):
    ragged = True           # runs ragged paged batches through ``forward_ragged`` (serve/engine.py)
    stateful = True         # keeps per-sequence states: the engine hands out state slots with the pages

    def __init__(self, cfg: KozasunConfig, *, dtype=torch.bfloat16, device=None):
        super().__init__()
        self.cfg, self.dtype = cfg, dtype
        self.embed = nn.Parameter(torch.empty(cfg.vocab_size, cfg.width, dtype=dtype, device=device))
        owners = [i for i, l in enumerate(cfg.layers) if l.owner == i]
        self.blocks = nn.ModuleList([KozasunBlock(cfg, cfg.layers[i], dtype, device) for i in owners])
        self.owners = owners                                               # layer index of every block's tensors
        self.runs = [owners.index(l.owner) for l in cfg.layers]            # block of every layer
        self.final_w = nn.Parameter(torch.ones(cfg.width, dtype=torch.float32, device=device))
        self.final_b = nn.Parameter(torch.zeros(cfg.width, dtype=torch.float32, device=device))
        self.head = nn.Parameter(torch.empty(cfg.vocab_size, cfg.width, dtype=dtype, device=device))
        self.final = hops.NextNorm(None, self.final_w, self.final_b)

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
            self.final_b.copy_(get("final.norm.b").float())
            for i, blk in zip(self.owners, self.blocks):
                blk.norm1.load(get, f"l{i}.", 1)
                blk.mixer.load(get, f"l{i}.mix.")
                if blk.mlp is not None:
                    blk.norm2.load(get, f"l{i}.", 2)
                    blk.mlp.load(get, f"l{i}.mlp.")

    def init_random(self, seed: int = 0) -> None:
        g = torch.Generator().manual_seed(seed)
        S = self.cfg.streams or 1
        with torch.no_grad():
            for name, p in self.named_parameters():
                leaf = name.rsplit(".", 1)[-1]
                if leaf in ("hc_in", "hc_out", "hc_mix"):
                    if self.cfg.streams is not None:
                        noise = torch.randn(p.shape, generator=g)
                        p.copy_(torch.eye(S) + 0.1 * noise / S if leaf == "hc_mix" else 1.0 / S + 0.1 * noise if leaf == "hc_in" else 1.0 + 0.1 * noise)
                elif leaf in ("bias", "b_in", "final_b", "correction"):
                    p.copy_((0.1 * torch.randn(p.shape, generator=g)).to(p.dtype))
                elif leaf == "sinks":
                    p.copy_(torch.randn(p.shape, generator=g))
                elif p.dim() == 1:
                    p.copy_((1.0 + 0.1 * torch.randn(p.shape, generator=g)).to(p.dtype))
                else:
                    p.copy_((torch.randn(p.shape, generator=g) / p.shape[-1] ** 0.5).to(p.dtype))

    # ---- caches and states -----------------------------------------------------------------------------
    def cache_bytes_per_block(self, block_size: int) -> int:
        it = torch.empty((), dtype=self.dtype).element_size()
        return sum(l.mixer.cache_width for l in self.cfg.layers if l.type != "retention") * block_size * it

    def allocate_caches(self, num_blocks: int, block_size: int, device, state_slots: int = 1) -> List[Any]:
        """One entry per layer (also for layers that share weights): the paged cache ``[pages, block_size, numbers per token]`` of an
        attention layer, the tuple of fp32 state tensors ``[state_slots, ...]`` of a retention layer."""
        def own(mixer: nn.Module) -> Any:
            if mixer.stateful:
                return tuple(torch.zeros(state_slots, *shape, dtype=torch.float32, device=device) for shape in mixer.state_shapes())
            return torch.zeros(mixer.cache_shape(num_blocks, block_size), dtype=self.dtype, device=device)
        return [own(self.blocks[b].mixer) for b in self.runs]

    # ---- forward ---------------------------------------------------------------------------------------
    @torch.no_grad()
    def forward_ragged(self, batch, caches: List[Any], layer_trace: Optional[list] = None) -> torch.Tensor:
        """``batch``: serve.ragged.RaggedBatch.  Returns fp32 logits [len(batch.out_rows), vocab]."""
        cfg, dt, eps = self.cfg, self.dtype, self.cfg.norm_eps
        blocks = [self.blocks[b] for b in self.runs]
        x, (h, h32) = hops.hyper_embed(batch.tokens, self.embed, cfg.embed_scale, cfg.streams or 1, blocks[0].norm1.nxt if blocks else None, eps)
        y = c = None            # output and stream weights of the last sublayer, whose update joins the output norm's pass
        for i, blk in enumerate(blocks):
            after = blocks[i + 1].norm1.nxt if i + 1 < len(blocks) else None
            y, c = blk.mixer(h, batch, caches[i]), blk.norm1.streams
            if blk.mlp is not None:
                h, h32 = hops.hyper_step(x, y, c, blk.norm2.nxt, eps, dt)
                y, c = blk.mlp(h, h32), blk.norm2.streams
            # the streams' update and the next layer's norm in one pass; the last one happens with the output norm, on wanted rows only
            if after is not None or layer_trace is not None:
                h, h32 = hops.hyper_step(x, y, c, after, eps, dt)
                if after is None:
                    y = c = None
            if layer_trace is not None:
                layer_trace.append(x.sum(1))
        if batch.num_out == 0:                  # a step that only fills the caches and states
            return torch.empty(0, cfg.vocab_size, dtype=torch.float32, device=x.device)
        z = hops.hyper_output(x, y, c, batch.out_rows, self.final, eps, dt)
        if z.is_cuda and dt == torch.bfloat16:
            if ops.kernel_config().gemm == "native" and ops._gemm_ok(z, self.head) and self.head.shape[0] % 8 == 0:
                return ops.gemm_raw(z, self.head, out_dtype=torch.float32)
            return torch.mm(z, self.head.t(), out_dtype=torch.float32)
        return torch.nn.functional.linear(z.float(), self.head.float())


def _load_weights(model: KozasunModel, directory) -> None:
    from safetensors.torch import load_file
    model.load_state(load_file(str(Path(directory) / "model.safetensors")))


def build_kozasun(cfg: KozasunConfig, *, dtype=torch.bfloat16, device=None, seed: int = 42, **_ignored) -> KozasunModel:
    m = KozasunModel(cfg, dtype=dtype, device=device)
    m.init_random(seed)
    return m


register_architecture(Architecture(name="Kozasun", config_from_dict=KozasunConfig.from_dict, config_type=KozasunConfig,
                                   build=build_kozasun, load_weights=_load_weights))


def example_config(width: int = 44, vocab: int = 70, pattern: str = "LARL", ff: str = "DMDM", shared_weights: Optional[Dict[int, int]] = None,
                   streams: Optional[int] = 2, heads: int = 4, kv_heads: int = 2, dim: int = 8, vdim: int = 6, rot_dims: int = 4,
                   rot_base: float = 500.0, att_scale: Optional[float] = None, chunk: int = 11, ret_heads: int = 3, ret_dim: int = 6,
                   ret_vdim: int = 10, ret_rot: int = 6, ret_base: float = 3000.0, decay: Optional[List[float]] = None, lat_heads: int = 3,
                   lat_dim: int = 5, lat_vdim: int = 7, kv_rank: int = 9, lat_scale: Optional[float] = None, window: int = 13, ff_size: int = 30,
                   experts: int = 6, top: int = 2, groups: Optional[tuple] = (3, 2), router_scale: float = 1.5, expert_ff: int = 14,
                   shared_ff: Optional[int] = 18, scale: float = 1.25, eps: float = 1e-5) -> Dict[str, Any]:
    """A small configuration dictionary for tests, benchmarks and examples.  ``pattern``: one character per layer for its mixer
    (A chunked attention, R retention, L latent attention); ``ff``: one character per layer for its feed-forward (D dense, M
    mixture of experts, - none), repeated; ``shared_weights``: {layer: layer whose weights it uses}."""
    layers: List[Dict[str, Any]] = []
    for i, ch in enumerate(pattern):
        if ch == "A":
            mixer: Dict[str, Any] = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk},
                                     "scale": dim ** -0.5 if att_scale is None else att_scale, "rot": {"base": rot_base, "dims": rot_dims}}
        elif ch == "R":
            rates = [1.0 - 2.0 ** (-2.0 - 4.0 * h / max(ret_heads - 1, 1)) for h in range(ret_heads)]
            mixer = {"heads": ret_heads, "dim": ret_dim, "vdim": ret_vdim, "decay": list(decay or rates), "rot": {"base": ret_base, "dims": ret_rot}}
        else:
            mixer = {"heads": lat_heads, "dim": lat_dim, "vdim": lat_vdim, "kv_rank": kv_rank, "mask": {"size": window},
                     "scale": lat_dim ** -0.5 if lat_scale is None else lat_scale}
        kind = ff[i % len(ff)]
        mlp: Optional[Dict[str, Any]] = None
        if kind == "D":
            mlp = {"kind": "dense", "ff": ff_size}
        elif kind == "M":
            router: Dict[str, Any] = {"experts": experts, "top": top, "scale": router_scale}
            if groups:
                router["groups"] = {"count": groups[0], "keep": groups[1]}
            mlp = {"kind": "moe", "router": router, "expert": {"ff": expert_ff}}
            if shared_ff:
                mlp["shared"] = {"ff": shared_ff}
        layers.append({"type": {"A": "attention", "R": "retention", "L": "latent_attention"}[ch], "mixer": mixer, "mlp": mlp})
    for i, j in (shared_weights or {}).items():
        layers[i] = {**layers[j], "weights_of": j}
    cfg: Dict[str, Any] = {"architecture": "Kozasun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale},
                           "layers": layers}
    if streams is not None:
        cfg["streams"] = streams
    return cfg
