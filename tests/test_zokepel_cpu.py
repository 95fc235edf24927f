"""Zokepel through the framework (op table, ragged batches, block manager with state slots, scheduler, engine) against the
plain oracle in ``zokepel_oracle.py``, on small random configurations.  These run on the CPU implementations of the ops;
``test_zokepel_gpu.py`` repeats the kernel-level and end-to-end comparisons on the CUDA kernels."""
import copy
import io
import json
import math

import pytest
import torch

import zokepel_oracle as oracle

F32 = 3e-4      # fp32 end to end against float64: rounding only


def make_engine(cfg, weights, dt=torch.float32, device="cpu", blocks=24, bs=8, max_batch=4, graphs=False):
    from llmctl_b200.serve.engine import InferenceEngine
    eng = InferenceEngine(copy.deepcopy(cfg), max_batch_size=max_batch, max_batch_tokens=blocks * bs, device=device,
                          kv_block_size=bs, num_kv_blocks=blocks, dtype=dt, kv_watermark=0.0, cuda_graphs=graphs)
    eng.model.load_state(weights)
    return eng


def small_cfg(**kw):
    from llmctl_b200.models.zokepel import example_config
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
    p = Portion(1, [0] * n_tokens, start, list(range(n_tokens)), table, 0)
    return RaggedBatch([p], bs, torch.device(device)), table


def portion_batch(n, at, slot=1, bs=64, device="cpu"):
    from llmctl_b200.serve.ragged import Portion, RaggedBatch
    return RaggedBatch([Portion(1, [0] * n, at, [], list(range((at + n + bs - 1) // bs)), slot)], bs, torch.device(device))


CONFIGS = {
    "default": dict(),
    "as_many_kv_heads_no_loop": dict(pattern="CDP", ff="111", loop=None, kv_heads=4, att_kv_heads=4, conv=4),
    "one_kv_head_no_ff": dict(pattern="PDC", ff="000", loop=(0, 3, 3), kv_heads=1, att_kv_heads=1, conv=2, vdim=3, att_vdim=5, q_temp=None),
    "ones": dict(pattern="CDP", ff="101", loop=(2, 3, 2), heads=1, kv_heads=1, dim=1, vdim=1, conv=1, decay_rank=1, gate_rank=1, att_heads=1,
                 att_kv_heads=1, att_dim=2, att_vdim=1, bias_rows=2, bias_max=3.0, mix_heads=1, mix_dim=1, mix_rank=1, q_temp=(0.7, 1)),
    "odd_sizes": dict(pattern="PCD", ff="010", loop=(1, 2, 2), width=36, heads=6, kv_heads=2, dim=7, vdim=9, conv=6, decay_rank=9, gate_rank=11,
                      att_heads=6, att_kv_heads=3, att_dim=5, att_vdim=7, bias_rows=12, bias_max=17.5, mix_heads=2, mix_dim=9, mix_rank=10,
                      limit=0.6, eps=1e-3, scale=0.5),
    "one_pass": dict(pattern="DP", ff="11", loop=(0, 2, 1), limit=4.0, bias_rows=6, bias_max=200.0),
}


# ---- mechanisms alone ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("W,scale", [(10, 2.5), (64, 0.3), (7, 1.0)])
def test_embedding_with_sinusoidal_positions(W, scale):
    from llmctl_b200.ops import dual_norm as D
    torch.manual_seed(W)
    table = torch.randn(9, W)
    toks = [3, 0, 8, 8, 1, 5]
    want = oracle.embedding(toks, table.double(), scale)
    x, copy_ = D.embed_sinusoid(torch.tensor(toks), torch.arange(6, dtype=torch.int32), table, scale, D.sinusoid_frequencies(W), want_copy=True)
    assert torch.allclose(x.double(), want, atol=1e-6) and torch.equal(x, copy_) and x.data_ptr() != copy_.data_ptr()
    # a far position: the angle is exact to fp32 rounding of its sine
    p = 123457
    x, none = D.embed_sinusoid(torch.tensor([2]), torch.tensor([p], dtype=torch.int32), table, 0.0, D.sinusoid_frequencies(W))
    assert none is None
    for c in range(W):
        a = p * 10000.0 ** (-2.0 * (c // 2) / W)
        assert abs(float(x[0, c]) - (math.sin(a) if c % 2 == 0 else math.cos(a))) < 1e-6


def test_residual_update_branch_sum_and_two_norms():
    from llmctl_b200.ops import dual_norm as D
    torch.manual_seed(0)
    T, W, eps = 5, 14, 1e-2
    x, a, b, f, e = (torch.randn(T, W) * s for s in (2.0, 0.1, 5.0, 1.0, 1.0))
    wa, wb, w1, w2 = (torch.rand(W) + 0.5 for _ in range(4))
    for m, f_, add in ((a, f, None), (D.BranchSum(a, b, wa, wb, 0.5), f, e), (D.BranchSum(a, b, wa, wb, 0.5), None, None), (None, None, e),
                       (a, None, e)):
        xs = x.clone()
        hs = D.residual_dual_norm(m, f_, xs, eps, [w1, w2], torch.float32, add=add)
        new = x.double()
        if isinstance(m, D.BranchSum):
            new = new + 0.5 * (oracle.rms(a.double(), eps) * wa.double() + oracle.rms(b.double(), eps) * wb.double())
        elif m is not None:
            new = new + a.double()
        new = new + (f.double() if f_ is not None else 0.0) + (e.double() if add is not None else 0.0)
        assert torch.allclose(xs.double(), new, atol=1e-6)
        for h, w in zip(hs, (w1, w2)):
            assert torch.allclose(h.double(), oracle.rms(new, eps) * w.double(), atol=1e-5)
    xs = x.clone()
    assert D.residual_dual_norm(a, None, xs, eps, [], torch.float32) == [] and torch.allclose(xs, x + a)
    assert len(D.residual_dual_norm(None, None, xs, eps, [w1], torch.float32)) == 1


def test_clamped_feed_forward():
    from llmctl_b200.models.ffn import GatedClampedMLP
    torch.manual_seed(1)
    P = {n: torch.randn(*s) for n, s in (("gate", (11, 8)), ("up", (11, 8)), ("down", (8, 11)))}
    mlp = GatedClampedMLP(8, 11, 0.8, 1.702, torch.float32, "cpu")
    mlp.load(lambda n: P[n], "")
    h = torch.randn(6, 8) * 2
    want = oracle.feed_forward(h.double(), {k: v.double() for k, v in P.items()}, 0.8)
    assert torch.allclose(mlp(h).double(), want, atol=1e-5)


@pytest.mark.parametrize("rows,far", [(8, 30.0), (16, 64.0), (32, 128.0), (2, 5.0), (6, 200.0), (12, 17.5), (10, 6.0), (64, 40.0)])
def test_distance_buckets(rows, far):
    """The table by distance against the bucket formula, at every distance past the last bucket's start."""
    from llmctl_b200.ops import softcap_attention as S
    rel = torch.arange(rows, dtype=torch.float32)[:, None].repeat(1, 2) + torch.tensor([0.0, 100.0])
    table = S.bucket_bias_table(rel, far)
    for n in range(int(far) + 40):
        b = oracle.bucket(n, rows, far)
        got = table[:, min(n, table.shape[1] - 1)]
        assert float(got[0]) == b and float(got[1]) == b + 100.0, (n, b, got)
    starts = S.distance_bucket_starts(rows, far)
    assert len(starts) == rows and starts[:rows // 2] == list(range(rows // 2)) and starts[rows // 2] == rows // 2


def attention_op(q, k, v, batch, cache, scale, table, H, G, d, e, bs, width):
    from llmctl_b200.ops import softcap_attention as S
    n = q.shape[0]
    tiles = torch.tensor([[s, min(width, n - s), 0, 0] for s in range(0, n, width)], dtype=torch.int32)
    return S.softcap_window_attention(q, cache, batch.block_tables, tiles, width, batch.positions, None, None, None, scale, 0.0, 0, 0, H, G, d,
                                      e, bs, torch.float32, table=table)


@pytest.mark.parametrize("H,G,d,e,n,bs,rows,far", [(4, 2, 8, 6, 45, 8, 8, 30.0), (3, 1, 5, 7, 33, 16, 4, 9.0), (2, 2, 4, 3, 50, 8, 2, 3.0),
                                                   (6, 3, 3, 2, 27, 4, 12, 17.5), (1, 1, 2, 1, 70, 64, 16, 200.0)])
def test_biased_attention_alone(H, G, d, e, n, bs, rows, far):
    from llmctl_b200.ops import softcap_attention as S
    torch.manual_seed(H * n)
    eps, coef, every = 1e-3, 0.6, 5
    q, k, v = torch.randn(n, H, d) * 3, torch.randn(n, G, d) * 0.2, torch.randn(n, G, e)
    rel = torch.randn(rows, H)
    batch, table = paged(n, bs, seed=n)
    cache = torch.zeros(len(table) + 3, bs, G * (d + e))
    proj = torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], dim=-1)
    qo = S.window_kv_append(proj, None, H, G, d, e, False, eps, batch.slots, cache, qk_norm=True, q_temp=(coef, every), positions=batch.positions)
    temp = torch.tensor([oracle.temperature(p, coef, every) for p in range(n)], dtype=torch.float64)[:, None, None]
    qn, kn = oracle.rms(q.double(), eps) * temp, oracle.rms(k.double(), eps)
    assert torch.allclose(qo.double(), qn.reshape(n, -1), atol=1e-5)
    want = oracle.biased_attention(qn, kn, v.double(), 0.4, rel.double(), far).reshape(n, -1)
    for width in (1, 16):
        got = attention_op(qo, k, v, batch, cache, 0.4, S.bucket_bias_table(rel, far), H, G, d, e, bs, width)
        assert torch.allclose(got.double(), want, atol=2e-6)


@pytest.mark.parametrize("bs,rows,far", [(8, 8, 30.0), (16, 4, 40.0), (4, 12, 17.5)])
def test_bias_bucket_edges_decide(bs, rows, far):
    """All scores are zero and one bucket's bias is large: the output is the mean value over exactly the keys in that bucket,
    so a bucket border that is one token off shows, within a page and at page borders."""
    from llmctl_b200.ops import softcap_attention as S
    n, e = int(far) + 30, 3
    torch.manual_seed(rows)
    v = torch.randn(n, 1, e)
    q = k = torch.zeros(n, 1, 2)
    batch, table = paged(n, bs, seed=rows)
    cache = torch.zeros(len(table) + 3, bs, 2 + e)
    qo = S.window_kv_append(torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], -1), None, 1, 1, 2, e, False, 0.0, batch.slots, cache)
    for star in range(rows):
        rel = torch.zeros(rows, 1)
        rel[star] = 40.0
        for width in (1, 16):
            out = attention_op(qo, k, v, batch, cache, 1.0, S.bucket_bias_table(rel, far), 1, 1, 2, e, bs, width)
            for i in range(n):
                seen = [j for j in range(i + 1) if oracle.bucket(i - j, rows, far) == star] or list(range(i + 1))
                assert torch.allclose(out[i], v[seen, 0].mean(0), atol=1e-5), (star, i)


@pytest.mark.parametrize("far_key,bs", [(0, 8), (7, 8), (8, 8), (63, 64), (64, 64)])
def test_far_key_decides(far_key, bs):
    """A key far back whose score stands out among ~200 others, at page borders, for prompt tiles and single tokens."""
    from llmctl_b200.ops import softcap_attention as S
    n, H, G, d, e = 210, 2, 1, 4, 3
    torch.manual_seed(far_key)
    q, k, v = torch.randn(n, H, d), torch.randn(n, G, d), torch.randn(n, G, e)
    q[-1] = torch.tensor([30.0, 0.0, 0.0, 0.0])
    k[:, :, 0] = -1.0
    k[far_key, :, 0] = 1.0
    rel = torch.randn(8, H)
    batch, table = paged(n, bs, seed=far_key)
    cache = torch.zeros(len(table) + 3, bs, d + e)
    qo = S.window_kv_append(torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], -1), None, H, G, d, e, False, 0.0, batch.slots, cache)
    want = oracle.biased_attention(q.double(), k.double(), v.double(), 1.0, rel.double(), 50.0).reshape(n, -1)
    for width in (1, 16):
        out = attention_op(qo, k, v, batch, cache, 1.0, S.bucket_bias_table(rel, 50.0), H, G, d, e, bs, width)
        assert torch.allclose(out.double(), want, atol=1e-5)
        assert torch.allclose(out[-1].view(H, e), v[far_key].expand(H, e), atol=1e-3)


@pytest.mark.parametrize("kind,H,G,d,e,taps,cuts", [("C", 4, 2, 6, 10, 3, [14]), ("C", 2, 2, 5, 3, 4, [2, 1, 1, 7, 2]), ("D", 6, 2, 4, 7, 2, [1] * 9),
                                                    ("D", 3, 1, 8, 8, 1, [5, 2, 6]), ("C", 1, 1, 1, 1, 5, [2, 2, 2, 3]), ("D", 4, 4, 3, 2, 7, [3, 1, 2, 8])])
def test_delta_rule_mixer_alone(kind, H, G, d, e, taps, cuts):
    """Both forms of the gated delta rule in portions (also shorter than the convolution), over a slot that holds garbage."""
    from llmctl_b200.models.zokepel import ZokepelConfig, ZokepelModel
    cfg = small_cfg(pattern=kind, ff="0", loop=None, heads=H, kv_heads=G, dim=d, vdim=e, conv=taps, width=16)
    w = oracle.random_weights(cfg, taps)
    mixer = ZokepelModel(ZokepelConfig.from_dict(cfg), dtype=torch.float32).blocks[0].mixer
    mixer.load(lambda n: w[n], "l0.mix.")
    torch.manual_seed(d)
    n = sum(cuts)
    h = torch.randn(n, 16)
    eps = cfg["norm"]["eps"]
    want = oracle.delta_mixer(h.double(), oracle.sub(w, "l0.mix."), cfg["layers"][0]["mixer"], eps, kind == "C")
    state = tuple(torch.full((3, *s), 5.0) for s in mixer.state_shapes())
    out, at = [], 0
    for c in cuts:
        out.append(mixer(h[at:at + c], portion_batch(c, at), state))
        at += c
    assert close(torch.cat(out), want, 2e-5)
    for s in state:                                     # the neighbours' slots are untouched
        assert torch.equal(s[[0, 2]], torch.full_like(s[[0, 2]], 5.0))


@pytest.mark.parametrize("H,d,rank,cuts", [(3, 5, 4, [13]), (2, 4, 1, [1] * 8), (1, 7, 9, [2, 1, 5, 2]), (4, 1, 3, [6, 2, 1, 1])])
def test_bonus_memory_mixer_alone(H, d, rank, cuts):
    from llmctl_b200.models.mixers import BonusMemory, BonusMemorySpec
    cfg = small_cfg(pattern="P", ff="0", loop=None, mix_heads=H, mix_dim=d, mix_rank=rank, width=16)
    w = oracle.random_weights(cfg, rank)
    eps = cfg["norm"]["eps"]
    mixer = BonusMemory(16, BonusMemorySpec(heads=H, dim=d, decay_rank=rank), eps, torch.float32, "cpu")
    mixer.load(lambda n: w[n], "l0.mix.right.")
    torch.manual_seed(d)
    h = torch.randn(sum(cuts), 16)
    want = oracle.right_mixer(h.double(), oracle.sub(w, "l0.mix.right."), cfg["layers"][0]["mixer"]["right"], eps)
    state = tuple(torch.full((2, *s), -3.0) for s in mixer.state_shapes())
    out, at = [], 0
    for c in cuts:
        out.append(mixer(h[at:at + c], portion_batch(c, at), state))
        at += c
    assert close(torch.cat(out), want, 2e-5)


def test_delta_rule_details_that_random_weights_hide():
    """A decay of one and full write strength: writing the same key twice replaces its value instead of adding to it (the
    delta), the read-out sees the current write, and a foreign key reads nothing."""
    d = e = 4
    eye = torch.eye(d, dtype=torch.float64)
    k = torch.stack([eye[0], eye[1], eye[0], eye[2]])[:, None]
    v = torch.tensor([[1.0, 0, 0, 0], [0, 2, 0, 0], [0, 0, 3, 0], [0, 0, 0, 4]], dtype=torch.float64)[:, None]
    q = torch.stack([eye[0], eye[0], eye[0], eye[3]])[:, None]
    one = torch.ones(4, 1, d, dtype=torch.float64)
    o = oracle.delta_rule(q, k, v, one, torch.ones(4, 1, dtype=torch.float64))[:, 0]
    assert torch.allclose(o, torch.stack([v[0, 0], v[0, 0], v[2, 0], torch.zeros(4, dtype=torch.float64)]))
    # the same numbers through the op: taps 1, silu inverted so that q, k, v come out as chosen up to the unit norm
    from llmctl_b200.ops import matrix_state as M

    def unsilu(y):
        z = torch.full_like(y, 1.0)
        for _ in range(200):
            s = torch.sigmoid(z)
            z = z - (z * s - y) / (s * (1 + z * (1 - s))).clamp_min(1e-3)
        return z
    raw = torch.cat([unsilu(q[:, 0] * 2), unsilu(k[:, 0] * 3), unsilu(v[:, 0])], dim=-1).float()
    state, conv = torch.full((1, 1, d, e), 9.0), torch.zeros(1, 0, 12)
    got = M.delta_rule(raw, torch.ones(12, 1), torch.full((4, 1), -60.0), torch.zeros(1), torch.ones(1), torch.full((4, 1), 60.0),
                       torch.full((4, e), 60.0), torch.ones(e), torch.tensor([[0, 4, 0, 0]], dtype=torch.int32), torch.zeros(4, dtype=torch.int32),
                       state, conv, 1, 1, d, e, False, 1e-9, "sigmoid")
    assert torch.allclose(got[:3].double(), oracle.rms(o[:3], 1e-9), atol=1e-4)
    assert torch.allclose(state[0, 0].double(), torch.stack([v[2, 0], v[1, 0], v[3, 0], torch.zeros(4, dtype=torch.float64)]), atol=1e-4)


def test_bonus_applies_to_the_current_token_only():
    """With a bonus and a key that never repeats: token t reads u k_t v_t now, and k_t v_t (without the bonus) later."""
    from llmctl_b200.ops import matrix_state as M
    T, d = 3, 2
    r = torch.tensor([[1.0, 0.0]]).repeat(T, 1)
    k = torch.tensor([[1.0, 0.0], [0.0, 1.0], [0.0, 0.0]])
    v = torch.tensor([[3.0, 4.0], [1.0, 1.0], [2.0, 2.0]])
    u = torch.tensor([7.0, 5.0])
    z = torch.full((T, d), math.log(0.5))             # decay exp(-0.5)
    state, shift = torch.zeros(1, 1, d, d), torch.zeros(1, d)
    M.bonus_memory(r, k, v, z, torch.zeros(d), u, torch.ones(T, d), torch.ones(d), torch.zeros(T, d), torch.tensor([[0, T, 0, 0]], dtype=torch.int32),
                   state, shift, 1, d, 1e-12)
    assert torch.allclose(state[0, 0], torch.stack([v[0] * math.exp(-1.0), v[1] * math.exp(-0.5)]), atol=1e-6)
    w = torch.full((T, 1, d), math.exp(-0.5), dtype=torch.float64)
    o = oracle.outer_memory(r[:, None].double(), k[:, None].double(), v[:, None].double(), w, u[None].double())[:, 0]
    assert torch.allclose(o[0], 7.0 * v[0].double()) and torch.allclose(o[1], v[0].double()) and torch.allclose(o[2], v[0].double() * math.exp(-0.5))


# ---- whole model ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_and_every_layer_run(name):
    cfg = small_cfg(**CONFIGS[name])
    w = oracle.random_weights(cfg, 11)
    toks = random_tokens(cfg, 29, 2)
    layers = []
    want = ref_logits(cfg, w, toks, layers)
    eng = make_engine(cfg, w)
    assert eng.kv.allocate(1, len(toks))
    trace = []
    got = eng.forward_portions([eng.portion(1, toks, 0, list(range(len(toks))))], layer_trace=trace)
    assert len(trace) == len(layers) == len(oracle.layer_order(cfg))
    for a, b in zip(trace, layers):
        assert close(a, b)
    assert close(got, want)
    eng2 = make_engine(cfg, w)                          # without the trace: the fused form of the glue
    assert close(run_cut(eng2, 1, toks, [29]), want)


@pytest.mark.parametrize("name,cuts", [("default", [1] * 26), ("default", [2, 2, 3, 2, 9, 1, 7]), ("odd_sizes", [5, 1, 2, 2, 16]),
                                       ("one_kv_head_no_ff", [13, 2, 2, 1, 8]), ("ones", [2, 1, 1, 1, 2, 19]),
                                       ("as_many_kv_heads_no_loop", [7, 19]), ("one_pass", [3, 2, 2, 20])])
def test_portions_against_whole_prompt(name, cuts):
    cfg = small_cfg(**CONFIGS[name])
    w = oracle.random_weights(cfg, 5)
    toks = random_tokens(cfg, sum(cuts), 3)
    assert close(run_cut(make_engine(cfg, w), 1, toks, cuts), ref_logits(cfg, w, toks))


def test_layers_of_one_kind_with_unlike_sizes():
    """Two layers of every kind, each pair with its own sizes, taps, ranks, scales, buckets and temperatures; a loop in the
    middle whose passes keep caches and states of their own."""
    a = small_cfg(pattern="CDP", ff="111")
    b = small_cfg(pattern="CDP", ff="101", heads=3, kv_heads=1, dim=5, vdim=4, conv=5, decay_rank=2, gate_rank=9, att_heads=6, att_kv_heads=1,
                  att_dim=4, att_vdim=6, att_scale=0.9, bias_rows=14, bias_max=90.0, q_temp=(0.2, 3), mix_heads=2, mix_dim=7, mix_rank=6,
                  ff_size=17, limit=0.5)
    cfg = copy.deepcopy(a)
    cfg["layers"] = [copy.deepcopy(l) for pair in zip(a["layers"], b["layers"]) for l in pair]
    cfg["loop"] = {"start": 1, "stop": 5, "times": 3}
    w = oracle.random_weights(cfg, 3)
    cuts = [7, 2, 20, 1, 1, 3, 16]
    toks = random_tokens(cfg, sum(cuts), 8)
    assert close(run_cut(make_engine(cfg, w), 1, toks, cuts), ref_logits(cfg, w, toks))


def test_unequal_batches_skipped_steps_and_reused_pages_and_slots():
    """Three seats and nine pages of 8 tokens for five requests of unequal length: portions of 1-11 tokens beside single tokens,
    requests that skip steps; pages and slots of finished requests go to the next ones.  Every position's logits equal the
    request's own whole-prompt logits."""
    cfg = small_cfg(pattern="CPD", ff="110", loop=(0, 2, 2))
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


def test_first_token_and_long_decoding_across_pages():
    """Slow decays: the first token still moves the last logits of a long decode; decoding runs token by token over many
    pages, past the last distance bucket and several temperature steps."""
    cfg = small_cfg(pattern="CDP", ff="111", loop=(0, 3, 2), bias_max=20.0, q_temp=(0.5, 16))
    w = oracle.random_weights(cfg, 3)
    for n in ("l0.mix.dt_bias", "l1.mix.dt_bias"):
        w[n] = torch.full_like(w[n], -9.0)
    w["l2.mix.right.w0"] = torch.full_like(w["l2.mix.right.w0"], -9.0)
    toks = random_tokens(cfg, 90, 8)
    want = ref_logits(cfg, w, toks)
    got = run_cut(make_engine(cfg, w), 1, toks, [10] + [1] * 80)
    assert close(got, want)
    other = ref_logits(cfg, w, [(toks[0] + 1) % cfg["vocab"]] + toks[1:])
    assert (other[-1] - want[-1]).abs().max() > 20 * F32


def test_greedy_generation_through_scheduler_and_engine():
    cfg = small_cfg(pattern="CPD", ff="111", loop=(1, 3, 2))
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
    """A checkpoint directory whose ``config.json`` names no ranks and no bias rows (the tensors' extents give them)."""
    import numpy as np
    from safetensors.torch import save_file
    from llmctl_b200.models.registry import architecture_named
    from llmctl_b200.models.zokepel import ZokepelConfig
    from llmctl_b200.serve import replay
    cfg = small_cfg(pattern="CPD", ff="110", loop=(0, 2, 2))
    w = oracle.random_weights(cfg, 2)
    bare = copy.deepcopy(cfg)
    for l in bare["layers"]:
        for m in (l["mixer"], l["mixer"].get("left", {}), l["mixer"].get("right", {})):
            for key in ("decay_rank", "gate_rank", "bias_rows"):
                m.pop(key, None)
    (tmp_path / "config.json").write_text(json.dumps(bare))
    save_file({k: v.to(torch.bfloat16) for k, v in w.items()}, str(tmp_path / "model.safetensors"))
    arch = architecture_named("Zokepel")
    parsed = arch.config_from_dict(bare)
    assert isinstance(parsed, ZokepelConfig) and [l.type for l in parsed.layers] == ["channel_delta", "parallel", "delta"]
    assert parsed.runs() == [(0, False), (1, False), (0, True), (1, False), (2, False)]
    arch.complete_config(parsed, tmp_path)
    assert parsed.layers[0].mixer.decay_rank == 5 and parsed.layers[0].mixer.gate_rank == 3
    assert parsed.layers[1].mixer.left.bias_rows == 8 and parsed.layers[1].mixer.right.decay_rank == 4 and parsed.layers[2].ff == 0
    for path, value in ((("loop", "stop"), 9), (("layers", 0, "type"), "other"), (("layers", 0, "mixer", "heads"), 3)):
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
