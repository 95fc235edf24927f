"""Kozasun through the framework (op table, ragged batches, block manager with state slots, scheduler, engine) against the
plain oracle in ``kozasun_oracle.py``, on small random configurations.  These run on the CPU implementations of the ops;
``test_kozasun_gpu.py`` repeats the kernel-level and end-to-end comparisons on the CUDA kernels."""
import copy
import io
import json

import pytest
import torch

import kozasun_oracle as oracle

F32 = 3e-4      # fp32 end to end against float64: rounding only
F64 = torch.float64


def make_engine(cfg, weights, dt=torch.float32, device="cpu", blocks=24, bs=8, max_batch=4, graphs=False):
    from llmctl_b200.serve.engine import InferenceEngine
    eng = InferenceEngine(copy.deepcopy(cfg), max_batch_size=max_batch, max_batch_tokens=blocks * bs, device=device,
                          kv_block_size=bs, num_kv_blocks=blocks, dtype=dt, kv_watermark=0.0, cuda_graphs=graphs)
    eng.model.load_state(weights)
    return eng


def small_cfg(**kw):
    from llmctl_b200.models.kozasun import example_config
    return example_config(**kw)


def ref_logits(cfg, w, toks, layers=None):
    return oracle.forward(cfg, w, toks, layers).float()


def close(got, want, tol=F32):
    return torch.allclose(got.float().cpu(), want.float(), atol=tol * max(1.0, float(want.abs().max())), rtol=0.0)


def random_tokens(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def run_cut(eng, sid, toks, cuts):
    """Feed ``toks`` in portions of the given sizes; returns logits of every position."""
    out, at = [], 0
    for c in cuts:
        assert eng.kv.allocate(sid, at + c)
        out.append(eng.forward_portions([eng.portion(sid, toks[at:at + c], at, list(range(c)))]))
        at += c
    assert at == len(toks)
    return torch.cat(out).float().cpu()


def paged(n_tokens, bs, device="cpu", start=0, seed=0):
    """A one-sequence ragged batch over shuffled pages: (batch, table)."""
    from llmctl_b200.serve.ragged import Portion, RaggedBatch
    nb = (start + n_tokens + bs - 1) // bs
    g = torch.Generator().manual_seed(seed)
    table = torch.randperm(nb + 3, generator=g)[:nb].tolist()
    return RaggedBatch([Portion(1, [0] * n_tokens, start, list(range(n_tokens)), table, 0)], bs, torch.device(device)), table


def portion_batch(n, at, slot=1, bs=64, device="cpu"):
    from llmctl_b200.serve.ragged import Portion, RaggedBatch
    return RaggedBatch([Portion(1, [0] * n, at, [], list(range((at + n + bs - 1) // bs)), slot)], bs, torch.device(device))


CONFIGS = {
    "default": dict(),
    "shared_weights": dict(pattern="LARALR", ff="MD", shared_weights={3: 1, 4: 0, 5: 2}, streams=3),
    "as_many_kv_heads_no_groups": dict(pattern="ARL", ff="M", kv_heads=4, groups=None, shared_ff=None, top=3, rot_dims=8, ret_rot=2, streams=4),
    "one_kv_head_no_ff": dict(pattern="RLA", ff="-", kv_heads=1, vdim=5, window=1, chunk=1, streams=1),
    "ones": dict(pattern="ALR", ff="MD-", heads=1, kv_heads=1, dim=2, vdim=1, rot_dims=2, ret_heads=1, ret_dim=2, ret_vdim=1, ret_rot=2, decay=[0.5],
                 lat_heads=1, lat_dim=1, lat_vdim=1, kv_rank=1, ff_size=1, experts=1, top=1, groups=None, expert_ff=1, shared_ff=1, streams=2),
    "odd_sizes": dict(width=37, vocab=53, pattern="LRAL", ff="MDM-", heads=6, kv_heads=3, dim=7, vdim=9, rot_dims=6, ret_heads=5, ret_dim=9, ret_vdim=7,
                      ret_rot=4, lat_heads=5, lat_dim=11, lat_vdim=3, kv_rank=13, ff_size=19, experts=10, top=4, groups=(5, 3), router_scale=0.7,
                      expert_ff=9, shared_ff=11, chunk=7, window=9, streams=5, scale=0.4, eps=1e-3),
    "groups_of_one": dict(pattern="RA", ff="M", experts=5, groups=(5, 3), top=3, router_scale=1.0, rot_dims=0, ret_rot=0),
    "one_stream_without_weights": dict(pattern="ALR", ff="DM", streams=None),
    "no_masks": dict(pattern="LA", ff="D", chunk=0, window=0),
}


def weights_for(cfg, seed):
    """Random checkpoint tensors, without stream weights for a configuration that names no streams (the oracle gets fixed ones)."""
    full = copy.deepcopy(cfg)
    full.setdefault("streams", 1)
    w = oracle.random_weights(full, seed)
    if "streams" in cfg:
        return full, w, w
    plain = {k: v for k, v in w.items() if ".hc" not in k}
    return full, plain, {k: (torch.ones_like(v) if ".hc" in k else v) for k, v in w.items()}


# ---- mechanisms alone ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("S,W", [(1, 6), (2, 9), (3, 16), (4, 5), (7, 8)])
def test_streams_and_layer_norm(S, W):
    """Embedding, updates that mix all streams from the old ones, next input, output over selected rows."""
    from llmctl_b200.ops import hyper_norm as H
    torch.manual_seed(S * W)
    T, eps, dt = 6, 1e-2, torch.float32
    table, toks = torch.randn(5, W), torch.tensor([4, 0, 2, 2, 1, 3])
    norms = [H.NextNorm(torch.randn(S), torch.rand(W) + 0.5, torch.randn(W), want_fp32=i == 1) for i in range(3)]
    final = H.NextNorm(None, torch.rand(W) + 0.5, torch.randn(W))
    steps = [H.StreamWeights(torch.zeros(S), torch.randn(S), torch.randn(S, S)) for _ in range(3)]
    ys = [torch.randn(T, W) for _ in range(3)]
    x, (h, h32) = H.hyper_embed(toks, table, 0.7, S, norms[0], eps)
    xs = torch.stack([table[toks].double() * 0.7] * S)
    assert x.shape == (T, S, W) and h32 is None

    def normed(n):
        u = sum((1.0 if n.a is None else n.a[s].double()) * xs[s] for s in range(S))
        return oracle.layer_norm(u, n.w.double(), n.bias.double(), eps)
    assert close(h, normed(norms[0]), 1e-5)
    for i in range(2):
        P = {"hc1.in": steps[i].a.double(), "hc1.out": steps[i].b.double(), "hc1.mix": steps[i].mix.double()}
        xs = oracle.hyper_step(xs, P, 1, lambda u: ys[i].double())
        h, h32 = H.hyper_step(x, ys[i], steps[i], norms[i + 1], eps, dt)
        assert close(x, xs.transpose(0, 1), 1e-5) and close(h, normed(norms[i + 1]), 1e-5)
        assert (h32 is not None) == norms[i + 1].want_fp32
    before = x.clone()
    rows = torch.tensor([5, 1, 1])
    assert close(H.hyper_output(x, None, None, rows, final, eps, dt), normed(final)[rows], 1e-5)
    P = {"hc1.in": steps[2].a.double(), "hc1.out": steps[2].b.double(), "hc1.mix": steps[2].mix.double()}
    xs = oracle.hyper_step(xs, P, 1, lambda u: ys[2].double())
    assert close(H.hyper_output(x, ys[2], steps[2], rows, final, eps, dt), normed(final)[rows], 1e-5) and torch.equal(x, before)
    H.hyper_step(x, ys[2], steps[2], None, eps, dt)
    assert close(x, xs.transpose(0, 1), 1e-5)


@pytest.mark.parametrize("H,G,d,e,rot,start", [(4, 2, 8, 6, 4, 0), (3, 1, 7, 5, 6, 100), (2, 2, 4, 3, 4, 9), (6, 3, 5, 1, 0, 3)])
def test_projection_norm_bias_and_rotated_halves(H, G, d, e, rot, start):
    from llmctl_b200.ops import window_attention as W
    from llmctl_b200.ops.elementwise import rope_frequencies
    torch.manual_seed(H * d)
    n, bs, eps = 9, 8, 1e-2
    base = 700.0
    proj, bias = torch.randn(n, H * d + G * (d + e) + 3), torch.randn(H * d + G * (d + e))
    qn, kn = torch.rand(H * d) + 0.5, torch.rand(G * d) + 0.5
    batch, table = paged(n, bs, start=start, seed=n)
    cache = torch.zeros(len(table) + 3, bs, G * (d + e))
    freq = rope_frequencies(rot, base)[0] if rot else torch.zeros(1)
    q = W.window_qkv_write(proj, bias, qn, kn, H, G, d, e, rot, freq, 1.0, eps, batch.positions, batch.slots, cache, bs, rot_half=True)
    f = proj[:, :H * d + G * (d + e)].double() + bias.double()
    pad = torch.zeros(start, 1, 1, dtype=F64)          # the oracle's rows are positions

    def turned(x, heads):
        x = torch.cat([pad.expand(start, heads, d), x.view(n, heads, d)])
        return oracle.rotate_halves(x, {"dims": rot, "base": base})[start:]
    wq = turned(oracle.rms(f[:, :H * d], eps) * qn.double(), H)
    wk = turned(oracle.rms(f[:, H * d:H * d + G * d], eps) * kn.double(), G)
    assert close(q, wq.reshape(n, -1), 1e-5)
    rows = cache.view(-1, G * (d + e))[batch.slots]
    assert close(rows[:, :G * d], wk.reshape(n, -1), 1e-5) and close(rows[:, G * d:], f[:, H * d + G * d:], 1e-5)


def attention_op(q, k, v, batch, cache, scale, sink, chunk, width, bs):
    """Fill the cache with given keys and values and attend; q: [n, H, d], k: [n, G, d], v: [n, G, e]."""
    from llmctl_b200.ops import softcap_attention as S
    n, H, d = q.shape
    G, e = v.shape[1], v.shape[2]
    qo = S.window_kv_append(torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], -1), None, H, G, d, e, False, 0.0, batch.slots, cache)
    tiles = torch.tensor([[s, min(width, n - s), 0, 0] for s in range(0, n, width)], dtype=torch.int32)
    return S.softcap_window_attention(qo, cache, batch.block_tables, tiles, width, batch.positions, None, None, sink, scale, 0.0, 0, 0, H, G, d, e,
                                      bs, torch.float32, chunk=chunk)


@pytest.mark.parametrize("H,G,d,e,n,bs,chunk", [(4, 2, 8, 6, 45, 8, 11), (3, 1, 5, 7, 33, 16, 16), (2, 2, 4, 3, 50, 8, 1), (6, 3, 3, 2, 27, 4, 40),
                                                (1, 1, 2, 1, 70, 64, 64), (2, 1, 4, 4, 30, 8, 0)])
def test_chunked_attention_with_sinks_alone(H, G, d, e, n, bs, chunk):
    torch.manual_seed(H * n)
    q, k, v, sink = torch.randn(n, H, d), torch.randn(n, G, d), torch.randn(n, G, e), torch.randn(H) * 2
    batch, table = paged(n, bs, seed=n)
    cache = torch.zeros(len(table) + 3, bs, G * (d + e))
    want = oracle.chunked_attention(q.double(), k.double(), v.double(), 0.4, chunk, sink.double()).reshape(n, -1)
    for width in (1, 16):
        assert torch.allclose(attention_op(q, k, v, batch, cache, 0.4, sink, chunk, width, bs).double(), want, atol=2e-6)


@pytest.mark.parametrize("bs,chunk", [(8, 11), (16, 16), (4, 6), (64, 33), (8, 24)])
def test_chunk_edges_decide(bs, chunk):
    """Equal scores and no weight on the sink: the output is the mean value over exactly the chunk's keys, so a border that is
    one token off shows, within a page and at page borders."""
    n, e = 3 * chunk + 2, 3
    torch.manual_seed(chunk)
    v = torch.randn(n, 1, e)
    zero = torch.zeros(n, 1, 2)
    batch, table = paged(n, bs, seed=chunk)
    cache = torch.zeros(len(table) + 3, bs, 2 + e)
    for width in (1, 16):
        out = attention_op(zero, zero, v, batch, cache, 1.0, torch.full((1,), -60.0), chunk, width, bs)
        for i in range(n):
            assert torch.allclose(out[i], v[i // chunk * chunk:i + 1, 0].mean(0), atol=1e-5), i


def test_sink_is_not_scaled_and_counts_once():
    """One key with score 0 and a sink of ln 3: the output is a quarter of the value whatever the scale; a very low sink leaves it."""
    v = torch.tensor([[[8.0]], [[8.0]]])
    zero = torch.zeros(2, 1, 2)
    for width in (1, 16):
        batch, table = paged(2, 8)
        cache = torch.zeros(len(table) + 3, 8, 3)
        out = attention_op(zero, zero, v, batch, cache, 0.01, torch.log(torch.tensor([3.0])), 4, width, 8)
        assert torch.allclose(out.reshape(-1), torch.tensor([2.0, 8.0 * 2 / 5]), atol=1e-5)
        out = attention_op(zero, zero, v, batch, cache, 0.01, torch.tensor([-80.0]), 4, width, 8)
        assert torch.allclose(out.reshape(-1), torch.tensor([8.0, 8.0]), atol=1e-5)


@pytest.mark.parametrize("key,bs", [(0, 8), (7, 8), (8, 8), (63, 64), (64, 64), (99, 8), (100, 8)])
def test_far_key_decides_within_its_chunk_only(key, bs):
    """A key whose score stands out among many others: it takes all the weight for queries of its chunk and none for others."""
    n, H, G, d, e, chunk = 210, 2, 1, 4, 3, 100
    torch.manual_seed(key)
    q, k, v = torch.randn(n, H, d), torch.randn(n, G, d), torch.randn(n, G, e)
    q[..., 0] = 30.0
    k[..., 0] = -1.0
    k[key, :, 0] = 1.0
    batch, table = paged(n, bs, seed=key)
    cache = torch.zeros(len(table) + 3, bs, d + e)
    sink = torch.zeros(H)
    want = oracle.chunked_attention(q.double(), k.double(), v.double(), 1.0, chunk, sink.double()).reshape(n, -1)
    end = (key // chunk + 1) * chunk
    for width in (1, 16):
        out = attention_op(q, k, v, batch, cache, 1.0, sink, chunk, width, bs)
        assert torch.allclose(out.double(), want, atol=1e-5)
        assert torch.allclose(out[end - 1].view(H, e), v[key].expand(H, e), atol=1e-3)
        assert not torch.allclose(out[end].view(H, e), v[key].expand(H, e), atol=1e-1)


def latent_op(ql, cache_rows, batch, table, scale, window, gate, width, bs):
    """ql: [n, H, R] absorbed queries; cache_rows: [n, R]."""
    from llmctl_b200.ops import latent_attention as L
    n, H, R = ql.shape
    cache = torch.zeros(len(table) + 3, bs, R)
    cache.view(-1, R)[batch.slots] = cache_rows
    tiles = torch.tensor([[s, min(width, n - s), 0, 0] for s in range(0, n, width)], dtype=torch.int32)
    return L.latent_attention(ql, torch.zeros(n, H), 1, cache, batch.block_tables, tiles, batch.positions, torch.zeros(1), 1.0, scale, H if width == 1 else 1,
                              n, rows=16, window=window, head_gate=gate)


@pytest.mark.parametrize("H,R,n,bs,window", [(3, 5, 40, 8, 13), (2, 8, 33, 16, 16), (1, 3, 20, 4, 1), (4, 6, 50, 8, 100), (2, 4, 30, 8, 0)])
def test_window_latent_attention_with_head_gates_alone(H, R, n, bs, window):
    torch.manual_seed(H * n)
    ql, c, gate = torch.randn(n, H, R), torch.randn(n, R), torch.randn(n, H)
    batch, table = paged(n, bs, seed=n)
    keys = c.double()[:, None, :].expand(n, H, R)
    want = oracle.window_attention(ql.double(), keys, keys, 0.3, window) * oracle.sigmoid(gate.double())[:, :, None]
    for width in (1, 16):
        assert torch.allclose(latent_op(ql, c, batch, table, 0.3, window, gate, width, bs).double(), want, atol=2e-6)


@pytest.mark.parametrize("bs,window", [(8, 11), (16, 16), (4, 1), (64, 33), (8, 24)])
def test_window_edges_decide(bs, window):
    """Zero queries: the output is the mean latent over exactly the window."""
    n, R = 3 * window + 5, 3
    torch.manual_seed(window)
    c = torch.randn(n, R)
    batch, table = paged(n, bs, seed=window)
    for width in (1, 16):
        out = latent_op(torch.zeros(n, 2, R), c, batch, table, 1.0, window, None, width, bs)
        for i in range(n):
            assert torch.allclose(out[i], c[max(i - window + 1, 0):i + 1].mean(0).expand(2, R), atol=1e-5), i


@pytest.mark.parametrize("H,d,e,rot,cuts", [(3, 6, 10, 6, [14]), (2, 5, 3, 2, [2, 1, 1, 7, 2]), (1, 2, 1, 0, [1] * 9), (4, 4, 8, 4, [5, 2, 6])])
def test_retention_mixer_alone(H, d, e, rot, cuts):
    """In portions, over a slot that holds garbage; the neighbours' slots are untouched."""
    from llmctl_b200.models.kozasun import KozasunConfig, KozasunModel
    cfg = small_cfg(pattern="R", ff="-", ret_heads=H, ret_dim=d, ret_vdim=e, ret_rot=rot, width=16)
    w = oracle.random_weights(cfg, d)
    mixer = KozasunModel(KozasunConfig.from_dict(cfg), dtype=torch.float32).blocks[0].mixer
    mixer.load(lambda n: w[n], "l0.mix.")
    torch.manual_seed(d)
    h = torch.randn(sum(cuts), 16)
    want = oracle.retention_mixer(h.double(), oracle.sub(w, "l0.mix."), cfg["layers"][0]["mixer"], cfg["norm"]["eps"])
    state = tuple(torch.full((3, *s), 5.0) for s in mixer.state_shapes())
    out, at = [], 0
    for c in cuts:
        out.append(mixer(h[at:at + c], portion_batch(c, at), state))
        at += c
    assert close(torch.cat(out), want, 2e-5)
    for s in state:
        assert torch.equal(s[[0, 2]], torch.full_like(s[[0, 2]], 5.0))


def test_retention_reads_its_own_write_and_decays_older_ones():
    """Unrotated unit keys: token t reads its own value at full weight, an older one times decay per step, keys times d^-1/2."""
    from llmctl_b200.ops import retention as R
    T, d, e = 4, 4, 2
    q = k = torch.tensor([[2.0, 0, 0, 0]]).repeat(T, 1)
    v = torch.tensor([[1.0, 0.0], [0.0, 1.0], [0.0, 0.0], [0.0, 0.0]])
    state = torch.full((1, 1, d, e), 7.0)
    decay = torch.tensor([-0.25])
    R.retention(q, k, v, torch.ones(T, e), torch.zeros(T, dtype=torch.int32), torch.zeros(1), 0, decay, torch.tensor([[0, T, 0, 0]], dtype=torch.int32), state,
                1, d, e, 1e-9)
    assert torch.allclose(state[0, 0, 0], torch.tensor([0.75 ** 3, 0.75 ** 2]), atol=1e-6) and state[0, 0, 1:].abs().max() == 0
    o = oracle.retention(q[:, None].double(), k[:, None].double() * d ** -0.5, v[:, None].double(), [0.75])[:, 0]
    assert torch.allclose(o[:2], torch.tensor([[2.0, 0.0], [1.5, 2.0]], dtype=F64))


@pytest.mark.parametrize("E,top,groups", [(6, 2, (3, 2)), (10, 4, (5, 3)), (8, 3, None), (5, 3, (5, 3)), (12, 2, (3, 1))])
def test_routing(E, top, groups):
    """Chosen experts and weights against the oracle's choice, most choice scores being negative."""
    from llmctl_b200.ops import moe as M
    torch.manual_seed(E)
    T, W = 40, 7
    x, wr, corr = torch.randn(T, W), torch.randn(E, W), torch.randn(E) * 0.5 - 0.8
    ids, wts, _, counts = M.route(x, wr, top, correction=corr, groups=groups, group_best=2, weight_scale=1.7)
    s = oracle.sigmoid(x.double() @ wr.double().T)
    for t in range(T):
        want = oracle.choose(s[t] + corr.double(), top, {"count": groups[0], "keep": groups[1]} if groups else None)
        assert sorted(ids[t].tolist()) == sorted(want)
        assert torch.allclose(wts[t].double(), s[t][ids[t].long()] * 1.7, atol=1e-6)
    assert int(counts.sum()) == T * top


def test_routing_group_is_worth_its_two_best():
    """The single best expert sits in a group that loses; the winners' scores are below it, and all choice scores are negative."""
    from llmctl_b200.ops import moe as M
    z = torch.tensor([[3.0, -9.0, 1.0, 1.0, 0.0, 0.5]])
    corr = torch.full((6,), -2.0)
    ids, wts, _, _ = M.route(z, torch.eye(6), 2, correction=corr, groups=(3, 1), group_best=2)
    assert sorted(ids[0].tolist()) == [2, 3] and torch.allclose(wts, torch.sigmoid(torch.tensor([[1.0, 1.0]])))
    ids, _, _, _ = M.route(z, torch.eye(6), 1, correction=corr, groups=(3, 1), group_best=1)
    assert ids[0].tolist() == [0]
    corr[5] = 1.0                                       # the correction chooses, the weight stays the plain score
    ids, wts, _, _ = M.route(z, torch.eye(6), 1, correction=corr, groups=(3, 1), group_best=2)
    assert ids[0].tolist() == [5] and torch.allclose(wts, torch.sigmoid(torch.tensor([[0.5]])))


# ---- whole model ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_and_every_layer(name):
    cfg = small_cfg(**CONFIGS[name])
    full, w, wo = weights_for(cfg, 11)
    toks = random_tokens(cfg, 29, 2)
    layers = []
    want = ref_logits(full, wo, toks, layers)
    eng = make_engine(cfg, w)
    assert eng.kv.allocate(1, len(toks))
    trace = []
    got = eng.forward_portions([eng.portion(1, toks, 0, list(range(len(toks))))], layer_trace=trace)
    assert len(trace) == len(layers) == len(cfg["layers"])
    for a, b in zip(trace, layers):
        assert close(a, b)
    assert close(got, want)
    eng2 = make_engine(cfg, w)                          # without the trace: the last update happens with the output norm
    assert close(run_cut(eng2, 1, toks, [29]), want)


@pytest.mark.parametrize("name,cuts", [("default", [1] * 30), ("default", [2, 2, 3, 2, 9, 1, 11]), ("odd_sizes", [5, 1, 2, 2, 16]),
                                       ("one_kv_head_no_ff", [13, 2, 2, 1, 8]), ("ones", [2, 1, 1, 1, 2, 19]), ("shared_weights", [7, 2, 1, 1, 19]),
                                       ("as_many_kv_heads_no_groups", [10, 1, 1, 12]), ("one_stream_without_weights", [3, 2, 2, 20])])
def test_portions_against_whole_prompt(name, cuts):
    cfg = small_cfg(**CONFIGS[name])
    full, w, wo = weights_for(cfg, 5)
    toks = random_tokens(cfg, sum(cuts), 3)
    assert close(run_cut(make_engine(cfg, w), 1, toks, cuts), ref_logits(full, wo, toks))


def test_layers_of_one_kind_with_unlike_sizes():
    """Two layers of every kind, each pair with its own sizes, masks, scales, rotations, decays and experts; a layer in front uses
    the weights of a later one."""
    a = small_cfg(pattern="LAR", ff="DMD", streams=3)
    b = small_cfg(pattern="LAR", ff="MDM", streams=3, heads=6, kv_heads=1, dim=4, vdim=9, rot_dims=2, rot_base=50.0, att_scale=0.9, chunk=5, ret_heads=2,
                  ret_dim=8, ret_vdim=3, ret_rot=4, decay=[0.3, 0.99], lat_heads=2, lat_dim=9, lat_vdim=4, kv_rank=17, lat_scale=0.2, window=6,
                  ff_size=11, experts=4, top=1, groups=(2, 1), router_scale=3.0, expert_ff=6, shared_ff=None)
    cfg = copy.deepcopy(a)
    cfg["layers"] = [copy.deepcopy(l) for pair in zip(a["layers"], b["layers"]) for l in pair]
    cfg["layers"].insert(0, {**copy.deepcopy(b["layers"][1]), "weights_of": 4})
    w = oracle.random_weights(cfg, 3)
    cuts = [7, 2, 20, 1, 1, 3, 16]
    toks = random_tokens(cfg, sum(cuts), 8)
    assert close(run_cut(make_engine(cfg, w), 1, toks, cuts), ref_logits(cfg, w, toks))


def test_unequal_batches_skipped_steps_and_reused_pages_and_slots():
    """Three seats and nine pages of 8 tokens for five requests of unequal length: portions of 1-11 tokens beside single tokens,
    requests that skip steps; pages and slots of finished requests go to the next ones.  Every position's logits equal the
    request's own whole-prompt logits."""
    cfg = small_cfg(pattern="LARA", ff="DMM", shared_weights={3: 1})
    w = oracle.random_weights(cfg, 9)
    lens = [30, 9, 17, 24, 5]
    prompts = [random_tokens(cfg, n, 40 + n) for n in lens]
    want = [ref_logits(cfg, w, p) for p in prompts]
    eng = make_engine(cfg, w, blocks=9, bs=8, max_batch=3)
    pos = [0] * len(prompts)
    got = [[] for _ in prompts]
    waiting, live, step = list(range(len(prompts))), [], 0
    sizes = [3, 1, 11, 2, 1, 1, 5]
    while waiting or live:
        while waiting and len(live) < 3 and eng.kv.allocate(waiting[0] + 1, min(sizes[0], lens[waiting[0]])):
            live.append(waiting.pop(0))
        portions, who = [], []
        for i in list(live):
            if (step + i) % 4 == 3:                     # this request sits the step out
                continue
            c = min(sizes[(step + 2 * i) % len(sizes)], lens[i] - pos[i])
            if not eng.kv.allocate(i + 1, pos[i] + c):
                continue                                # no page free right now: wait for somebody to finish
            portions.append(eng.portion(i + 1, prompts[i][pos[i]:pos[i] + c], pos[i], list(range(c))))
            who.append((i, c))
            pos[i] += c
        if portions:
            lg, o = eng.forward_portions(portions).float(), 0
            for i, c in who:
                got[i].append(lg[o:o + c])
                o += c
        for i in list(live):
            if pos[i] == lens[i]:
                eng.kv.free(i + 1)
                live.remove(i)
        step += 1
        assert step < 500
    for i in range(len(prompts)):
        assert close(torch.cat(got[i]), want[i]), i


def test_steps_that_want_nothing_fill_caches_and_states():
    cfg = small_cfg()
    w = oracle.random_weights(cfg, 6)
    toks = random_tokens(cfg, 20, 1)
    eng = make_engine(cfg, w)
    for at, c in ((0, 9), (9, 1), (10, 9)):
        assert eng.kv.allocate(1, at + c)
        assert eng.forward_portions([eng.portion(1, toks[at:at + c], at, [])]).shape == (0, cfg["vocab"])
    assert eng.kv.allocate(1, 20)
    assert close(eng.forward_portions([eng.portion(1, toks[19:], 19, [0])]), ref_logits(cfg, w, toks)[-1:])


def test_first_token_and_long_decoding_across_pages():
    """Slow decays: the first token still moves the last logits through the retention alone (window and chunk are far behind);
    decoding runs token by token over many pages, windows and chunks."""
    cfg = small_cfg(pattern="RLA", ff="DM", decay=[0.999, 0.9999, 0.5], window=9, chunk=10)
    w = oracle.random_weights(cfg, 3)
    toks = random_tokens(cfg, 90, 8)
    want = ref_logits(cfg, w, toks)
    assert close(run_cut(make_engine(cfg, w), 1, toks, [10] + [1] * 80), want)
    other = ref_logits(cfg, w, [(toks[0] + 1) % cfg["vocab"]] + toks[1:])
    assert (other[-1] - want[-1]).abs().max() > 20 * F32


@pytest.mark.parametrize("layer,size", [("A", 16), ("A", 11), ("L", 16), ("L", 13)])
def test_one_layer_model_sees_exactly_its_mask(layer, size):
    """A model of one attention layer: changing a token moves the logits at exactly the positions that see it, in prompts and in
    decoding."""
    cfg = small_cfg(pattern=layer, ff="-", chunk=size, window=size)
    w = oracle.random_weights(cfg, size)
    n = 3 * size + 1
    toks = random_tokens(cfg, n, 4)
    for at in (0, size - 1, size, 2 * size - 1, 2 * size):
        changed = list(toks)
        changed[at] = (toks[at] + 1) % cfg["vocab"]
        sees = [i >= at and (i // size == at // size if layer == "A" else i - at < size) for i in range(n)]
        for cuts in ([n], [size + 3] + [1] * (n - size - 3)):
            a, b = (run_cut(make_engine(cfg, w), 1, t, cuts) for t in (toks, changed))
            moved = [(a[i] - b[i]).abs().max() > 1e-4 for i in range(n)]
            assert moved == sees, (at, cuts[0])


def test_greedy_generation_through_scheduler_and_engine():
    cfg = small_cfg(pattern="LARL", ff="MD", streams=3)
    w = oracle.random_weights(cfg, 21)
    prompts = [random_tokens(cfg, n, n) for n in (5, 12, 3, 9, 7)]
    eng = make_engine(cfg, w, blocks=16, bs=8, max_batch=2)             # more requests than seats
    outs = eng.generate(prompts, max_tokens=6, temperature=0.0)
    for p, o in zip(prompts, outs):
        seq = list(p)
        for _ in range(6):
            seq.append(int(ref_logits(cfg, w, seq)[-1].argmax()))
        assert list(o) == seq[len(p):]


def test_config_reader_registry_and_trace_replay(tmp_path):
    import numpy as np
    from safetensors.torch import save_file
    from llmctl_b200.models.kozasun import KozasunConfig
    from llmctl_b200.models.registry import architecture_named
    from llmctl_b200.serve import replay
    cfg = small_cfg(pattern="LARA", ff="MD", shared_weights={3: 1}, streams=3)
    w = oracle.random_weights(cfg, 2)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.to(torch.bfloat16) for k, v in w.items()}, str(tmp_path / "model.safetensors"))
    arch = architecture_named("Kozasun")
    parsed = arch.config_from_dict(cfg)
    assert isinstance(parsed, KozasunConfig) and [l.type for l in parsed.layers] == ["latent_attention", "attention", "retention", "attention"]
    assert [l.owner for l in parsed.layers] == [0, 1, 2, 1] and parsed.streams == 3 and parsed.to_dict() == cfg
    assert parsed.num_parameters() == sum(v.numel() for v in w.values()) + _padding(parsed)
    for path, value in ((("layers", 0, "type"), "other"), (("layers", 1, "mixer", "kv_heads"), 3), (("layers", 2, "mixer", "decay"), [0.5]),
                        (("layers", 3, "weights_of"), 2), (("layers", 3, "weights_of"), 3), (("layers", 1, "mixer", "rot", "dims"), 3),
                        (("streams",), 0), (("layers", 0, "mlp", "kind"), "other")):
        bad = copy.deepcopy(cfg)
        at = bad
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            arch.config_from_dict(bad)
    a, b = random_tokens(cfg, 21, 6), random_tokens(cfg, 10, 7)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:9], "want": [8]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[9:11], "want": []}, {"id": "b", "tokens": b[:7], "want": [0, 6]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[7:], "want": [2]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[11:], "want": [9]}], "end": ["a"]}]
    out = io.StringIO()
    rc = replay.run(str(tmp_path), "float32", str(tmp_path / "out"), 128, device="cpu", stdin=io.StringIO("\n".join(json.dumps(s) for s in steps)),
                    stdout=out)
    assert rc == 0 and out.getvalue().split() == ["done", "0", "done", "1", "done", "2", "done", "3"]
    la, lb = ref_logits(cfg, w, a), ref_logits(cfg, w, b)

    def rd(s):
        return torch.from_numpy(np.fromfile(tmp_path / "out" / f"{s}.f32", dtype="<f4").reshape(-1, cfg["vocab"]))
    assert close(rd(0), la[[8]]) and close(rd(1), lb[[0, 6]]) and close(rd(2), lb[[9]]) and close(rd(3), la[[20]])


def _padding(parsed) -> int:
    """Rows of zeros that the packed projections add (parts start at multiples of 8)."""
    def up(n):
        return (n + 7) // 8 * 8 - n
    rows = 0
    for i, l in enumerate(parsed.layers):
        m = l.mixer
        if l.owner != i or l.type == "attention":
            continue
        parts = (m.heads * m.dim, m.heads * m.dim, m.heads * m.vdim, m.heads * m.vdim) if l.type == "retention" else (m.kv_rank, m.heads * m.dim, m.heads)
        rows += sum(up(n) for n in parts)
    return rows * parsed.width
