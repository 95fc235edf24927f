"""A plain, slow restatement of the Kozasun design in float64, for tests: whole sequences, no cache, no state slots, no
batching, one function per mechanism.  It shares no code with the package.

Streams:  s copies of the scaled embedding; per sublayer u = sum_s a_s x_s, y = f(layernorm(u)),
          x_t <- sum_s M[s, t] x_s + b_t y; at the end the streams are added up
Mixers:   chunked softmax attention (projection norms, rotated halves, a sink per head); retention (a fixed decay per head);
          latent attention over a sliding window with a gate per head
Feed-forward: gated GELU, or routed gated-SiLU experts chosen within the best groups, beside a shared one."""
from __future__ import annotations

import math
from typing import Any, Dict, List, Optional

import torch

F64 = torch.float64


def rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def layer_norm(v: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    c = v - v.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w + b


def silu(z: torch.Tensor) -> torch.Tensor:
    return z / (1.0 + torch.exp(-z))


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def gelu(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate_halves(x: torch.Tensor, rot: Optional[Dict[str, Any]]) -> torch.Tensor:
    """x: [T, heads, d], the row index being the position; coordinate i turns with coordinate i + dims / 2."""
    if not rot or not rot["dims"]:
        return x
    n, half = rot["dims"], rot["dims"] // 2
    out = x.clone()
    for p in range(x.shape[0]):
        for i in range(half):
            a = p * float(rot["base"]) ** (-2.0 * i / n)
            u, v = x[p, :, i], x[p, :, i + half]
            out[p, :, i] = u * math.cos(a) - v * math.sin(a)
            out[p, :, i + half] = v * math.cos(a) + u * math.sin(a)
    return out


def chunked_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, chunk: int, sink: torch.Tensor) -> torch.Tensor:
    """q: [T, H, d]; k: [T, G, d]; v: [T, G, e]; sink: [H].  Position i sees the keys of its own chunk up to itself."""
    T, H = q.shape[0], q.shape[1]
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for i in range(T):
        lo = i // chunk * chunk if chunk else 0
        for h in range(H):
            s = (k[lo:i + 1, h // rep] @ q[i, h]) * scale
            top = torch.maximum(s.max(), sink[h])
            w = torch.exp(s - top)
            out[i, h] = (w / (w.sum() + torch.exp(sink[h] - top))) @ v[lo:i + 1, h // rep]
    return out


def attention_mixer(h: torch.Tensor, P: Dict[str, torch.Tensor], m: Dict[str, Any], eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(h @ P["q"].T + P["q.b"], eps) * P["q.norm"]
    k = rms(h @ P["k"].T + P["k.b"], eps) * P["k.norm"]
    v = h @ P["v"].T + P["v.b"]
    q, k = rotate_halves(q.view(T, H, d), m["rot"]), rotate_halves(k.view(T, G, d), m["rot"])
    return chunked_attention(q, k, v.view(T, G, e), m["scale"], m["mask"]["size"], P["sink"]).reshape(T, H * e) @ P["o"].T


def retention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: List[float]) -> torch.Tensor:
    """q, k: [T, H, d]; v: [T, H, e]; the read-out sees the token's own write.  Returns [T, H, e]."""
    T, H, d = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        s = torch.zeros(d, v.shape[2], dtype=F64)
        for t in range(T):
            s = decay[h] * s + k[t, h][:, None] * v[t, h][None, :]
            out[t, h] = s.T @ q[t, h]
    return out


def retention_mixer(h: torch.Tensor, P: Dict[str, torch.Tensor], m: Dict[str, Any], eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d, e = m["heads"], m["dim"], m["vdim"]
    q = rotate_halves((h @ P["q"].T).view(T, H, d), m["rot"])
    k = rotate_halves((h @ P["k"].T).view(T, H, d), m["rot"]) * d ** -0.5
    o = rms(retention(q, k, (h @ P["v"].T).view(T, H, e), m["decay"]), eps)
    return (o.reshape(T, H * e) * silu(h @ P["g"].T)) @ P["o"].T


def window_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window: int) -> torch.Tensor:
    """q, k: [T, H, d]; v: [T, H, e].  Position i sees itself and the window - 1 keys before it."""
    T, H = q.shape[0], q.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for i in range(T):
        lo = max(i - window + 1, 0) if window else 0
        for h in range(H):
            out[i, h] = torch.softmax((k[lo:i + 1, h] @ q[i, h]) * scale, 0) @ v[lo:i + 1, h]
    return out


def latent_mixer(h: torch.Tensor, P: Dict[str, torch.Tensor], m: Dict[str, Any], eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d, e = m["heads"], m["dim"], m["vdim"]
    c = rms(h @ P["dkv"].T, eps) * P["dkv.norm"]
    q, k, v = (h @ P["q"].T).view(T, H, d), (c @ P["uk"].T).view(T, H, d), (c @ P["uv"].T).view(T, H, e)
    o = window_attention(q, k, v, m["scale"], m["mask"]["size"]) * sigmoid(h @ P["g"].T)[:, :, None]
    return o.reshape(T, H * e) @ P["o"].T


MIXERS = {"attention": attention_mixer, "retention": retention_mixer, "latent_attention": latent_mixer}


def choose(choice: torch.Tensor, top: int, groups: Optional[Dict[str, int]]) -> List[int]:
    """Expert indices for one token: the largest choice scores within the groups whose two best scores add up to most."""
    E = choice.numel()
    allowed = list(range(E))
    if groups:
        n = E // groups["count"]
        value = [sum(sorted(choice[g * n:(g + 1) * n].tolist(), reverse=True)[:2]) for g in range(groups["count"])]
        kept = sorted(range(groups["count"]), key=lambda g: -value[g])[:groups["keep"]]
        allowed = [e for e in range(E) if e // n in kept]
    return sorted(allowed, key=lambda e: -float(choice[e]))[:top]


def gated(h: torch.Tensor, P: Dict[str, torch.Tensor], p: str, act) -> torch.Tensor:
    return (act(h @ P[p + "gate"].T) * (h @ P[p + "up"].T)) @ P[p + "down"].T


def feed_forward(h: torch.Tensor, P: Dict[str, torch.Tensor], mlp: Dict[str, Any]) -> torch.Tensor:
    if mlp["kind"] == "dense":
        return gated(h, P, "", gelu)
    r = mlp["router"]
    score = sigmoid(h @ P["router"].T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in choose(score[t] + P["correction"], r["top"], r.get("groups")):
            out[t] += score[t, e] * r["scale"] * gated(h[t:t + 1], P, f"e{e}.", silu)[0]
    if mlp.get("shared"):
        out = out + gated(h, P, "shared.", silu)
    return out


def hyper_step(xs: torch.Tensor, P: Dict[str, torch.Tensor], q: int, f) -> torch.Tensor:
    """One sublayer on the streams xs [s, T, W]; f maps the mixed input to the sublayer's output."""
    a, b, m = P[f"hc{q}.in"], P[f"hc{q}.out"], P[f"hc{q}.mix"]
    n = xs.shape[0]
    y = f(sum(a[s] * xs[s] for s in range(n)))
    return torch.stack([sum(m[s, t] * xs[s] for s in range(n)) + b[t] * y for t in range(n)])


def sub(tensors: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v.to(F64) for k, v in tensors.items() if k.startswith(prefix)}


def owner(cfg: Dict[str, Any], i: int) -> int:
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg: Dict[str, Any], tensors: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] (float64) of one whole sequence; ``layers_out`` collects the sum of the streams after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = tensors["embed"].to(F64)[torch.tensor(tokens)] * float(cfg["embedding"]["scale"])
    xs = torch.stack([x] * cfg["streams"])
    for i, layer in enumerate(cfg["layers"]):
        P = sub(tensors, f"l{owner(cfg, i)}.")
        mix, mlp = sub(P, "mix."), sub(P, "mlp.")
        xs = hyper_step(xs, P, 1, lambda u: MIXERS[layer["type"]](layer_norm(u, P["norm1"], P["norm1.b"], eps), mix, layer["mixer"], eps))
        if layer.get("mlp") is not None:
            xs = hyper_step(xs, P, 2, lambda u: feed_forward(layer_norm(u, P["norm2"], P["norm2.b"], eps), mlp, layer["mlp"]))
        if layers_out is not None:
            layers_out.append(xs.sum(0))
    return layer_norm(xs.sum(0), tensors["final.norm"].to(F64), tensors["final.norm.b"].to(F64), eps) @ tensors["head"].to(F64).T


def random_weights(cfg: Dict[str, Any], seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random checkpoint tensors (float32 values that bfloat16 holds exactly) for a configuration dictionary."""
    g = torch.Generator().manual_seed(seed)
    W, S = cfg["width"], cfg["streams"]

    def rnd(v):
        return v.to(torch.bfloat16).float()

    def mat(o, i, s=1.0):
        return rnd(torch.randn(o, i, generator=g) * s / i ** 0.5)

    def vec(n, mean=0.0, s=1.0):
        return rnd(mean + s * torch.randn(n, generator=g))
    t: Dict[str, torch.Tensor] = {"embed": mat(cfg["vocab"], W, 3.0), "head": mat(cfg["vocab"], W), "final.norm": vec(W, 1.0, 0.1),
                                  "final.norm.b": vec(W, 0.0, 0.2)}
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        m, mlp, p = layer["mixer"], layer.get("mlp"), f"l{i}.mix."
        for q in (1, 2) if mlp is not None else (1,):
            t[f"l{i}.norm{q}"], t[f"l{i}.norm{q}.b"] = vec(W, 1.0, 0.1), vec(W, 0.0, 0.2)
            t[f"l{i}.hc{q}.in"], t[f"l{i}.hc{q}.out"] = vec(S, 0.6, 0.3), vec(S, 0.8, 0.4)
            t[f"l{i}.hc{q}.mix"] = rnd(0.7 * torch.eye(S) + 0.3 * torch.randn(S, S, generator=g) / S)
        H, d, e = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            G = m["kv_heads"]
            for s, rows in (("q", H * d), ("k", G * d), ("v", G * e)):
                t[p + s], t[p + s + ".b"] = mat(rows, W), vec(rows, 0.0, 0.3)
            t[p + "q.norm"], t[p + "k.norm"], t[p + "sink"] = vec(H * d, 1.0, 0.2), vec(G * d, 1.0, 0.2), vec(H)
        elif layer["type"] == "retention":
            t[p + "q"], t[p + "k"], t[p + "v"], t[p + "g"] = mat(H * d, W), mat(H * d, W), mat(H * e, W), mat(H * e, W)
        else:
            R = m["kv_rank"]
            t[p + "q"], t[p + "dkv"], t[p + "dkv.norm"] = mat(H * d, W), mat(R, W), vec(R, 1.0, 0.2)
            t[p + "uk"], t[p + "uv"], t[p + "g"] = mat(H * d, R), mat(H * e, R), mat(H, W)
        t[p + "o"] = mat(W, H * e)
        p = f"l{i}.mlp."
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            t[p + "gate"], t[p + "up"], t[p + "down"] = mat(mlp["ff"], W), mat(mlp["ff"], W), mat(W, mlp["ff"])
            continue
        E = mlp["router"]["experts"]
        t[p + "router"], t[p + "correction"] = mat(E, W), vec(E, -0.4, 0.4)
        for s, ff in [(f"e{k}.", mlp["expert"]["ff"]) for k in range(E)] + ([("shared.", mlp["shared"]["ff"])] if mlp.get("shared") else []):
            t[p + s + "gate"], t[p + s + "up"], t[p + s + "down"] = mat(ff, W), mat(ff, W), mat(W, ff)
    return t
