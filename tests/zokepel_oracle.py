"""A plain, slow restatement of the Zokepel design in float64, for tests: whole sequences, no cache, no state slots, no
batching, one function per mechanism.  It shares no code with the package.

Layer:   x <- x + mixer(rms(x) w1) + ff(rms(x) w2)
Loop:    layers start .. stop-1 run `times` times; the embedding output joins the stream before every pass but the first
Mixers:  gated delta rule with a decay per key channel or per head; softmax attention (normed queries and keys, query
         temperature, bucketed distance bias) beside a decayed outer-product memory over token-shifted inputs."""
from __future__ import annotations

import math
from typing import Any, Dict, List, Optional

import torch

F64 = torch.float64


def rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z / (1.0 + torch.exp(-z))


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.log1p(torch.exp(-z.abs())) + z.clamp_min(0.0)


def embedding(tokens: List[int], table: torch.Tensor, scale: float) -> torch.Tensor:
    """Scaled rows plus sines (even entries) and cosines (odd entries) of position times a falling frequency."""
    W = table.shape[1]
    x = table[torch.tensor(tokens)] * scale
    for p in range(len(tokens)):
        for c in range(W):
            angle = p * 10000.0 ** (-2.0 * (c // 2) / W)
            x[p, c] += math.sin(angle) if c % 2 == 0 else math.cos(angle)
    return x


def short_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x: [T, C]; w: [C, taps], the last tap multiplies the current token; followed by silu."""
    T, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += w[:, j] * x[s]
    return silu(out)


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor) -> torch.Tensor:
    """q, k: [T, G, d] unit vectors (q already scaled); v: [T, H, e]; g: [T, H, d] decays; beta: [T, H].  Returns [T, H, e]."""
    T, H, e = v.shape
    G, d = k.shape[1], k.shape[2]
    out = torch.zeros(T, H, e, dtype=F64)
    for h in range(H):
        s = torch.zeros(d, e, dtype=F64)
        kv = h // (H // G)
        for t in range(T):
            s = g[t, h][:, None] * s
            u = beta[t, h] * (v[t, h] - s.T @ k[t, kv])
            s = s + k[t, kv][:, None] * u[None, :]
            out[t, h] = s.T @ q[t, kv]
    return out


def delta_mixer(h: torch.Tensor, P: Dict[str, torch.Tensor], m: Dict[str, Any], eps: float, channels: bool) -> torch.Tensor:
    """channels: the decay has one number per head and key channel (low-rank projection) and the output gate is a sigmoid;
    otherwise one number per head and a silu gate."""
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit(short_conv(h @ P["q"].T, P["q.conv"]).view(T, G, d)) * d ** -0.5
    k = unit(short_conv(h @ P["k"].T, P["k.conv"]).view(T, G, d))
    v = short_conv(h @ P["v"].T, P["v.conv"]).view(T, H, e)
    beta = torch.sigmoid(h @ P["b"].T)
    speed = torch.exp(P["A_log"])
    if channels:
        step = softplus((h @ P["a1"].T) @ P["a2"].T + P["dt_bias"]).view(T, H, d)
        g = torch.exp(-speed[None, :, None] * step)
        gate = torch.sigmoid((h @ P["g1"].T) @ P["g2"].T)
    else:
        step = softplus(h @ P["a"].T + P["dt_bias"])
        g = torch.exp(-speed[None, :] * step)[:, :, None].expand(T, H, d)
        gate = silu(h @ P["g"].T)
    o = rms(delta_rule(q, k, v, g, beta), eps) * P["norm"]
    return (o.reshape(T, H * e) * gate) @ P["o"].T


def bucket(n: int, rows: int, far: float) -> int:
    half = rows // 2
    if n < half:
        return n
    # the logarithm's steps: bucket half + s begins where (n / half)^(rows - half) reaches (far / half)^s
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half) + 1e-12))


def biased_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, rel: torch.Tensor, far: float) -> torch.Tensor:
    """q: [T, H, d]; k: [T, G, d]; v: [T, G, e]; rel: [rows, H].  Returns [T, H, e]."""
    T, H = q.shape[0], q.shape[1]
    rep = H // k.shape[1]
    table = torch.stack([rel[bucket(n, rel.shape[0], far)] for n in range(T)])           # [T, H] by distance
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for i in range(T):
        dist = i - torch.arange(i + 1)
        for h in range(H):
            s = (k[:i + 1, h // rep] @ q[i, h]) * scale + table[dist, h]
            out[i, h] = torch.softmax(s, 0) @ v[:i + 1, h // rep]
    return out


def temperature(p: int, coef: float, every: float) -> float:
    return 1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0)


def left_mixer(h: torch.Tensor, P: Dict[str, torch.Tensor], m: Dict[str, Any], eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ P["q"].T).view(T, H, d), eps)
    k = rms((h @ P["k"].T).view(T, G, d), eps)
    v = (h @ P["v"].T).view(T, G, e)
    if m.get("q_temp"):
        q = q * torch.tensor([temperature(p, m["q_temp"]["coef"], m["q_temp"]["every"]) for p in range(T)], dtype=F64)[:, None, None]
    return biased_attention(q, k, v, m["scale"], P["rel"], m["bias_max"]).reshape(T, H * e) @ P["o"].T


def outer_memory(r: torch.Tensor, k: torch.Tensor, v: torch.Tensor, w: torch.Tensor, u: torch.Tensor) -> torch.Tensor:
    """r, k, v, w: [T, H, d]; u: [H, d].  The read-out sees the state before the token plus the token's own bonus."""
    T, H, d = r.shape
    out = torch.zeros(T, H, d, dtype=F64)
    for h in range(H):
        s = torch.zeros(d, d, dtype=F64)
        for t in range(T):
            kv = k[t, h][:, None] * v[t, h][None, :]
            out[t, h] = (s + u[h][:, None] * kv).T @ r[t, h]
            s = w[t, h][:, None] * s + kv
    return out


def right_mixer(h: torch.Tensor, P: Dict[str, torch.Tensor], m: Dict[str, Any], eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    before = torch.cat([torch.zeros(1, h.shape[1], dtype=F64), h[:-1]])
    mix = {s: h + (before - h) * P["mu." + s] for s in "rkvgw"}
    r, k, v = ((mix[s] @ P[s].T).view(T, H, d) for s in "rkv")
    w = torch.exp(-torch.exp(torch.tanh(mix["w"] @ P["w1"].T) @ P["w2"].T + P["w0"])).view(T, H, d)
    o = rms(outer_memory(r, k, v, w, P["u"]), eps).reshape(T, H * d) * P["norm"]
    return (o * silu(mix["g"] @ P["g"].T)) @ P["o"].T


def parallel_mixer(h: torch.Tensor, P: Dict[str, torch.Tensor], m: Dict[str, Any], eps: float) -> torch.Tensor:
    left, right = sub(P, "left."), sub(P, "right.")
    return 0.5 * (rms(left_mixer(h, left, m["left"], eps), eps) * left["out"] + rms(right_mixer(h, right, m["right"], eps), eps) * right["out"])


def feed_forward(h: torch.Tensor, P: Dict[str, torch.Tensor], limit: float) -> torch.Tensor:
    g = (h @ P["gate"].T).clamp(max=limit)
    u = (h @ P["up"].T).clamp(-limit, limit)
    return (g / (1.0 + torch.exp(-1.702 * g)) * (u + 1.0)) @ P["down"].T


def sub(tensors: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v.to(F64) for k, v in tensors.items() if k.startswith(prefix)}


def layer_order(cfg: Dict[str, Any]) -> List[tuple]:
    """(layer, the embedding output joins before it) of every layer run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, t = loop["start"], loop["stop"], loop["times"]
    order = [(i, False) for i in range(a)]
    for p in range(t):
        order += [(i, p > 0 and i == a) for i in range(a, b)]
    return order + [(i, False) for i in range(b, n)]


def forward(cfg: Dict[str, Any], tensors: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] (float64) of one whole sequence; ``layers_out`` collects the stream after every layer run."""
    eps = float(cfg["norm"]["eps"])
    x0 = embedding(tokens, tensors["embed"].to(F64), float(cfg["embedding"]["scale"]))
    x = x0.clone()
    for i, rejoin in layer_order(cfg):
        layer = cfg["layers"][i]
        if rejoin:
            x = x + x0
        n, P, m = rms(x, eps), sub(tensors, f"l{i}.mix."), layer["mixer"]
        h1 = n * tensors[f"l{i}.norm1"].to(F64)
        if layer["type"] == "parallel":
            y = parallel_mixer(h1, P, m, eps)
        else:
            y = delta_mixer(h1, P, m, eps, layer["type"] == "channel_delta")
        if layer.get("mlp") is not None:
            y = y + feed_forward(n * tensors[f"l{i}.norm2"].to(F64), sub(tensors, f"l{i}.mlp."), float(layer["mlp"]["limit"]))
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return (rms(x, eps) * tensors["final.norm"].to(F64)) @ tensors["head"].to(F64).T


def random_weights(cfg: Dict[str, Any], seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random checkpoint tensors (float32 values that bfloat16 holds exactly) for a configuration dictionary that also names the
    sizes which a checkpoint's tensors give (ranks of the low-rank projections, rows of the bias table)."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def rnd(v):
        return v.to(torch.bfloat16).float()

    def mat(o, i, s=1.0):
        return rnd(torch.randn(o, i, generator=g) * s / i ** 0.5)

    def vec(n, mean=0.0, s=1.0):
        return rnd(mean + s * torch.randn(n, generator=g))

    def uni(n, lo, hi):
        return rnd(lo + (hi - lo) * torch.rand(n, generator=g))
    t: Dict[str, torch.Tensor] = {"embed": mat(cfg["vocab"], W), "head": mat(cfg["vocab"], W), "final.norm": vec(W, 1.0, 0.1)}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        t[f"l{i}.norm1"] = vec(W, 1.0, 0.1)
        if layer["type"] == "parallel":
            a, r = m["left"], m["right"]
            H, G, d, e = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            t[p + "left.q"], t[p + "left.k"], t[p + "left.v"] = mat(H * d, W), mat(G * d, W), mat(G * e, W)
            t[p + "left.rel"], t[p + "left.o"] = rnd(torch.randn(a["bias_rows"], H, generator=g)), mat(W, H * e)
            H, d = r["heads"], r["dim"]
            for s in "rkvgw":
                t[p + "right.mu." + s] = uni(W, 0.0, 1.0)
            for s in "rkvg":
                t[p + "right." + s] = mat(H * d, W)
            t[p + "right.w1"], t[p + "right.w2"], t[p + "right.w0"] = mat(r["decay_rank"], W), mat(H * d, r["decay_rank"]), uni(H * d, -6.0, 0.5)
            t[p + "right.u"], t[p + "right.norm"] = rnd(torch.randn(H, d, generator=g)), vec(H * d, 1.0, 0.1)
            t[p + "right.o"] = mat(W, H * d)
            t[p + "left.out"], t[p + "right.out"] = vec(W, 1.0, 0.1), vec(W, 1.0, 0.1)
        else:
            H, G, d, e, c = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for s, rows in (("q", G * d), ("k", G * d), ("v", H * e)):
                t[p + s], t[p + s + ".conv"] = mat(rows, W), mat(rows, c, 1.5)
            t[p + "b"], t[p + "A_log"], t[p + "norm"] = mat(H, W), uni(H, -2.0, 1.0), vec(e, 1.0, 0.1)
            if layer["type"] == "channel_delta":
                t[p + "a1"], t[p + "a2"], t[p + "dt_bias"] = mat(m["decay_rank"], W), mat(H * d, m["decay_rank"]), uni(H * d, -5.0, 0.0)
                t[p + "g1"], t[p + "g2"] = mat(m["gate_rank"], W), mat(H * e, m["gate_rank"])
            else:
                t[p + "a"], t[p + "dt_bias"], t[p + "g"] = mat(H, W), uni(H, -5.0, 0.0), mat(H * e, W)
            t[p + "o"] = mat(W, H * e)
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            t[f"l{i}.norm2"] = vec(W, 1.0, 0.1)
            t[f"l{i}.mlp.gate"], t[f"l{i}.mlp.up"], t[f"l{i}.mlp.down"] = mat(ff, W), mat(ff, W), mat(W, ff)
    return t
