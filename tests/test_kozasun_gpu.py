"""Kozasun's CUDA kernels against the CPU restatements of the same ops and the engine on a GPU against the plain oracle
(``kozasun_oracle.py``), in fp32 (tight) and bf16 (rounding-sized)."""
import pytest
import torch

import kozasun_oracle as oracle
from test_kozasun_cpu import CONFIGS, make_engine, paged, random_tokens, ref_logits, run_cut, small_cfg, weights_for

pytestmark = pytest.mark.gpu


def rel(a, b):
    """Largest row error: rms of the difference (mean taken off) over the rms of the reference row."""
    d = a.double().cpu() - b.double().cpu()
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / b.double().cpu().pow(2).mean(-1).sqrt().clamp_min(1e-9)).max())


# number of streams with a kernel of its own and beyond, widths on the 16-byte and the scalar path, few and many rows
@pytest.mark.parametrize("S,T,W", [(1, 5, 10), (2, 33, 37), (3, 7, 320), (4, 3, 2048), (5, 9, 64), (9, 4, 30), (3, 2, 9000), (4, 400, 96)])
def test_stream_kernels(cuda_device, S, T, W):
    from llmctl_b200.ops import hyper_norm as H
    torch.manual_seed(S * W)
    dev = cuda_device
    g = lambda t: None if t is None else t.to(dev)  # noqa: E731

    def both(f):
        return f(lambda t: t), f(g)
    a, b, mix = torch.randn(S), torch.randn(S), torch.randn(S, S)
    w, bias = torch.rand(W) + 0.5, torch.randn(W)
    toks = torch.randint(0, 11, (T,))
    rows = torch.tensor([T - 1, 0, 0])
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 3e-2)):
        table = torch.randn(11, W).to(dt)
        for ydt in {torch.float32, dt}:
            y = torch.randn(T, W + 8).to(ydt)[:, :W]
            for want32 in (False, True):
                def chain(mv):
                    nxt = H.NextNorm(mv(a), mv(w), mv(bias), want32)
                    x, (h0, h0f) = H.hyper_embed(mv(toks), mv(table), 0.7, S, nxt, 1e-4)
                    c = H.StreamWeights(mv(a), mv(b), mv(mix))
                    out = [x.clone(), h0, h0f]
                    for _ in range(2):
                        out += [*H.hyper_step(x, mv(y), c, nxt, 1e-4, dt), x.clone()]
                    out.append(H.hyper_output(x, mv(y), c, mv(rows), H.NextNorm(None, mv(w), mv(bias)), 1e-4, dt))
                    out.append(H.hyper_output(x, None, None, mv(rows), H.NextNorm(None, mv(w), mv(bias)), 1e-4, dt))
                    H.hyper_step(x, mv(y), c, None, 1e-4, dt)
                    return out + [x]
                for u, v in zip(*both(chain)):
                    assert (u is None) == (v is None)
                    if u is not None:
                        s = max(1.0, float(u.float().abs().max()))
                        assert u.dtype == v.dtype and torch.allclose(v.float().cpu(), u.float(), atol=(tol if u.dtype == dt else 2e-5) * s, rtol=1e-2 if u.dtype != torch.float32 else 0)


@pytest.mark.parametrize("H,G,d,e,rot", [(4, 2, 8, 6, 4), (3, 1, 7, 5, 6), (8, 2, 64, 40, 32), (6, 3, 20, 12, 20), (2, 2, 128, 128, 64), (4, 1, 6, 3, 0)])
@pytest.mark.parametrize("half", [False, True])
def test_projection_append_kernel(cuda_device, H, G, d, e, rot, half):
    from llmctl_b200.ops import window_attention as W
    from llmctl_b200.ops.elementwise import rope_frequencies
    dev = cuda_device
    torch.manual_seed(H * d)
    n, bs, start = 37, 16, 700
    N = H * d + G * (d + e)
    freq = rope_frequencies(rot, 5000.0)[0] if rot else torch.zeros(1)
    bc, table = paged(n, bs, start=start, seed=n)
    bg, _ = paged(n, bs, device=dev, start=start, seed=n)
    qn, kn = torch.rand(H * d) + 0.5, torch.rand(G * d) + 0.5
    for dt, tol in ((torch.float32, 2e-5), (torch.bfloat16, 3e-2)):
        for extra, bdt, norm in ((0, torch.float32, True), (5, dt, True), (8, None, False)):
            proj = torch.randn(n, N + extra).to(dt)
            bias = torch.randn(N).to(bdt) if bdt is not None else None
            cc = torch.zeros(len(table) + 3, bs, G * (d + e), dtype=dt)
            cg = cc.to(dev)
            args = (H, G, d, e, rot)
            qc = W.window_qkv_write(proj, bias, qn if norm else None, kn if norm else None, *args, freq, 1.0, 1e-4, bc.positions, bc.slots, cc, bs,
                                    rot_half=half)
            qg = W.window_qkv_write(proj.to(dev), None if bias is None else bias.to(dev), qn.to(dev) if norm else None, kn.to(dev) if norm else None, *args,
                                    freq.to(dev), 1.0, 1e-4, bg.positions, bg.slots, cg, bs, rot_half=half)
            assert torch.allclose(qg.cpu(), qc, atol=3e-4) and torch.allclose(cg.float().cpu(), cc.float(), atol=3e-4 + (tol if dt != torch.float32 else 0.0))


@pytest.mark.parametrize("H,G,d,e,n,bs,chunk", [(4, 2, 8, 6, 45, 16, 11), (3, 1, 5, 7, 133, 16, 50), (8, 2, 16, 16, 300, 64, 120), (8, 4, 48, 40, 200, 64, 33),
                                                (4, 4, 32, 64, 150, 8, 1), (16, 2, 128, 128, 290, 64, 200), (2, 1, 16, 136, 70, 16, 64), (6, 6, 64, 72, 400, 64, 131)])
def test_chunked_attention_kernels(cuda_device, H, G, d, e, n, bs, chunk):
    """FMA and tensor-core kernels: prompt tiles, single tokens, key slices; a prompt and a later portion of it."""
    from llmctl_b200.ops import softcap_attention as S
    dev = cuda_device
    torch.manual_seed(H * d)
    q, sink = torch.randn(n, H * d), torch.randn(H)
    bc, pages = paged(n, bs, seed=n)
    bg, _ = paged(n, bs, device=dev, seed=n)
    for dt, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
        cc = torch.randn(len(pages) + 3, bs, G * (d + e)).to(dt)
        cg = cc.to(dev)
        t16 = torch.tensor([[s, min(16, n - s), 0, 0] for s in range(0, n, 16)], dtype=torch.int32)
        args = (d ** -0.5, 0.0, 0, 0, H, G, d, e, bs, dt)
        want = S.softcap_window_attention(q, cc, bc.block_tables, t16, 16, bc.positions, None, None, sink, *args, chunk=chunk)
        for width, splits, mma in ((16, 0, False), (1, 1, False), (1, 3, False), (128, 0, True), (1, 1, True), (1, 4, True)):
            if mma and not S.uses_tensor_cores(dt, H, G, d, e, width):
                continue
            for first in (0, n // 3):
                tiles = torch.tensor([[s, min(width, n - s), 0, 0] for s in range(first, n, width)], dtype=torch.int32)
                got = S.softcap_window_attention(q.to(dev), cg, bg.block_tables, tiles.to(dev), width, bg.positions, None, None, sink.to(dev), *args,
                                                 max_context=n, splits=splits, tensor_cores=mma, chunk=chunk)
                assert torch.allclose(got.float().cpu()[first:], want.float()[first:], atol=tol, rtol=1e-2), (dt, width, splits, mma, first)


@pytest.mark.parametrize("d,e,chunk", [(16, 8, 33), (6, 5, 16), (16, 8, 100)])
def test_chunk_edges_decide(cuda_device, d, e, chunk):
    """Equal scores: the output is the mean value of exactly the chunk's keys so far (fp32 and bf16 kernels)."""
    from llmctl_b200.ops import softcap_attention as S
    dev, n, bs = cuda_device, 310, 16
    torch.manual_seed(d)
    i = torch.arange(n)
    seen = (i[:, None] >= i[None, :]) & (i[:, None] // chunk == i[None, :] // chunk)
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        batch, pages = paged(n, bs, device=dev, seed=3)
        v = torch.randn(n, e).to(dt)
        cache = torch.zeros(len(pages) + 3, bs, d + e, dtype=dt, device=dev)
        cache.view(-1, d + e)[batch.slots, d:] = v.to(dev)
        want = (seen.double() / seen.double().sum(-1, keepdim=True)) @ v.double()
        for width in (1, 16, 128):
            if width == 128 and not S.uses_tensor_cores(dt, 1, 1, d, e, width):
                continue
            tiles = torch.tensor([[s, min(width, n - s), 0, 0] for s in range(0, n, width)], dtype=torch.int32, device=dev)
            out = S.softcap_window_attention(torch.zeros(n, d, device=dev), cache, batch.block_tables, tiles, width, batch.positions, None, None,
                                             torch.full((1,), -60.0, device=dev), 1.0, 0.0, 0, 0, 1, 1, d, e, bs, dt, max_context=n, chunk=chunk)
            assert torch.allclose(out.double().cpu(), want, atol=tol), (dt, width)


# latent sizes for the FMA kernel, the mma.sync kernel and (multiples of 64) the tcgen05 kernel
@pytest.mark.parametrize("H,R,n,bs,window", [(3, 10, 70, 16, 13), (2, 48, 200, 64, 64), (5, 64, 300, 64, 100), (20, 64, 150, 64, 1), (4, 128, 260, 64, 136),
                                             (3, 512, 200, 64, 90), (6, 192, 290, 32, 0), (33, 80, 90, 64, 41)])
def test_window_latent_attention_kernels(cuda_device, H, R, n, bs, window):
    from llmctl_b200.ops import latent_attention as L
    dev = cuda_device
    torch.manual_seed(H * R)
    bc, pages = paged(n, bs, seed=n)
    bg, _ = paged(n, bs, device=dev, seed=n)
    ql, gate = torch.randn(H, n, R) * 2 / R ** 0.5, torch.randn(n, H + 3)[:, 3:]
    fr = torch.zeros(1)
    for dt, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
        cc = torch.randn(len(pages) + 3, bs, R).to(dt)
        gt = gate.to(dt)
        t16 = torch.tensor([[s, min(16, n - s), 0, 0] for s in range(0, n, 16)], dtype=torch.int32)
        q = torch.zeros(n, H, dtype=dt)
        qd = ql.to(dt).float() if dt == torch.bfloat16 and L.uses_tensor_cores(dt, R, 0) else ql
        want = L.latent_attention(qd.transpose(0, 1), q, 1, cc, bc.block_tables, t16, bc.positions, fr, 1.0, 0.8, 1, n, rows=16, window=window, head_gate=gt)
        for width, splits, rows in ((16, 1, 16), (1, 1, 16), (1, 3, 16), (32, 1, 32), (1, 2, 32), (128, 1, 128), (128, 2, 128)):
            tc = dt == torch.bfloat16 and L.uses_tensor_cores(dt, R, 0)
            if rows == 32 and L.rows_per_tile(dt, R, 0, True) != 32 or rows == 128 and not L.uses_tcgen05(dt, R, 0, bs, True):
                continue
            for first in (0, n // 3):
                tiles = torch.tensor([[s, min(width, n - s), 0, 0] for s in range(first, n, width)], dtype=torch.int32).to(dev)
                qg = qd.to(dev).to(torch.bfloat16) if tc else qd.to(dev)
                got = L.latent_attention(qg.transpose(0, 1), q.to(dev), 1, cc.to(dev), bg.block_tables, tiles, bg.positions, fr.to(dev), 1.0, 0.8,
                                         min(H, rows) if width == 1 else 1, n, splits=splits, rows=rows, window=window, head_gate=gt.to(dev))
                assert torch.allclose(got.float().cpu()[first:], want.float()[first:], atol=tol, rtol=1e-2), (dt, width, splits, rows, first)
    assert not hasattr(L, "tcgen05_status") or L.tcgen05_status() == 0


@pytest.mark.parametrize("R,window", [(10, 33), (48, 16), (64, 100), (64, 32), (128, 65)])
def test_window_edges_decide(cuda_device, R, window):
    """Zero queries: the output is the mean latent of exactly the window, on every kernel that takes the sizes."""
    from llmctl_b200.ops import latent_attention as L
    dev, n, bs, H = cuda_device, 310, 64, 2
    torch.manual_seed(R)
    i = torch.arange(n)
    dist = i[:, None] - i[None, :]
    seen = ((dist >= 0) & (dist < window)).double()
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        batch, pages = paged(n, bs, device=dev, seed=3)
        c = torch.randn(n, R).to(dt)
        cache = torch.zeros(len(pages) + 3, bs, R, dtype=dt, device=dev)
        cache.view(-1, R)[batch.slots] = c.to(dev)
        want = (seen / seen.sum(-1, keepdim=True)) @ c.double()
        for width, rows in ((1, 16), (16, 16), (32, 32), (128, 128)):
            if rows == 32 and L.rows_per_tile(dt, R, 0, True) != 32 or rows == 128 and not L.uses_tcgen05(dt, R, 0, bs, True):
                continue
            tiles = torch.tensor([[s, min(width, n - s), 0, 0] for s in range(0, n, width)], dtype=torch.int32, device=dev)
            tc = dt == torch.bfloat16 and L.uses_tensor_cores(dt, R, 0)
            ql = torch.zeros(H, n, R, device=dev, dtype=torch.bfloat16 if tc else torch.float32)
            out = L.latent_attention(ql.transpose(0, 1), torch.zeros(n, H, dtype=dt, device=dev), 1, cache, batch.block_tables, tiles, batch.positions,
                                     torch.zeros(1, device=dev), 1.0, 1.0, H if width == 1 else 1, n, rows=rows, window=window)
            assert torch.allclose(out.double().cpu(), want[:, None].expand(n, H, R), atol=tol), (dt, width, rows)


def portions_of(lens, pos, slots, device="cpu"):
    starts = [sum(lens[:i]) for i in range(len(lens))]
    p = torch.tensor([[starts[i], lens[i], pos[i], slots[i]] for i in range(len(lens))], dtype=torch.int32)
    positions = torch.tensor(sum((list(range(pos[i], pos[i] + n)) for i, n in enumerate(lens)), []), dtype=torch.int32)
    return p.to(device), positions.to(device)


# sizes on every padded row count and beside it, odd and vector-aligned value sizes, several column blocks
@pytest.mark.parametrize("H,d,e,rot", [(4, 6, 10, 4), (2, 32, 32, 32), (3, 40, 36, 20), (4, 64, 100, 64), (2, 128, 128, 128), (3, 97, 33, 0), (2, 256, 64, 64),
                                       (1, 1, 1, 0), (2, 128, 256, 64), (2, 64, 128, 32), (5, 48, 80, 16),
                                       (2, 16, 256, 8), (1, 112, 224, 104)])
def test_retention_kernels(cuda_device, H, d, e, rot):
    """Prompts of unequal lengths side by side (one without a slot, one at position 0 over garbage), then decoding steps by the
    single-launch kernel, all from the same evolving states."""
    from llmctl_b200.ops import retention as R
    from llmctl_b200.ops.elementwise import rope_frequencies
    torch.manual_seed(H * d + e)
    dev = cuda_device
    nk, nv = H * d, H * e
    freq = rope_frequencies(rot, 3000.0)[0] if rot else torch.zeros(1)
    decay = -torch.rand(H) * torch.tensor([0.3, 0.01, 0.001, 0.1, 0.9][:H])
    for dt, tol in ((torch.float32, 1e-4), (torch.bfloat16, 2e-2)):
        st = torch.randn(4, H, d, e)
        sg = st.clone().to(dev)
        pos, slots = [5, 0, 9], [2, 0, -1]
        for lens in ([19, 137, 3], [2, 1, 16], [1, 1, 1], [1, 1, 1], [73, 1, 2], [1, 1, 1], [64, 65, 63], [2, 330, 128]):
            p = torch.randn(sum(lens), 2 * nk + 2 * nv + (8 if (nk + nv) % 8 == 0 else 3)).to(dt)
            po, ps = portions_of(lens, pos, slots)

            tiles = torch.tensor([[sum(lens[:i]) + s, min(R.CHUNK, n - s), i, 0] for i, n in enumerate(lens) for s in range(0, n, R.CHUNK)],
                                 dtype=torch.int32)

            def run(p, po, ps, st, dev, tiles=None):
                q, k, v, g = (p[:, a:b] for a, b in ((0, nk), (nk, 2 * nk), (2 * nk, 2 * nk + nv), (2 * nk + nv, 2 * nk + 2 * nv)))
                return R.retention(q, k, v, g, ps.to(dev), freq.to(dev), rot, decay.to(dev), po.to(dev), st, H, d, e, 1e-2, decode=max(lens) == 1,
                                   tiles=tiles)
            before = sg.clone()
            want = run(p, po, ps, st, "cpu")
            for tl in (None, tiles.to(dev)):                # the serial scan, then (bf16, sizes allowing) chunks on the tensor cores
                sg.copy_(before)
                got = run(p.to(dev), po, ps, sg, dev, tl)
                assert got.dtype == dt and torch.allclose(got.float().cpu(), want.float(), atol=tol * max(1.0, float(want.float().abs().max())), rtol=0), lens
                assert torch.allclose(sg.cpu(), st, atol=(5e-5 if dt == torch.float32 else 2e-4) * max(1.0, float(st.abs().max()))), lens
            pos = [a + b for a, b in zip(pos, lens)]


@pytest.mark.parametrize("E,top,groups,best", [(6, 2, (3, 2), 2), (10, 4, (5, 3), 2), (8, 3, None, 2), (5, 3, (5, 3), 2), (64, 6, (8, 3), 2), (64, 6, (8, 3), 1)])
def test_routing_kernel(cuda_device, E, top, groups, best):
    from llmctl_b200.ops import moe as M
    torch.manual_seed(E)
    T, W = 90, 36
    x, wr, corr = torch.randn(T, W), torch.randn(E, W) / W ** 0.5, torch.randn(E) * 0.5 - 0.8
    for dt in (torch.float32, torch.bfloat16):
        a = M.route(x, wr.to(dt), top, correction=corr, groups=groups, group_best=best, weight_scale=1.7)
        b = M.route(x.cuda(), wr.to(dt).cuda(), top, correction=corr.cuda(), groups=groups, group_best=best, weight_scale=1.7)
        ia, ib = a[0].sort(-1), b[0].cpu().sort(-1)
        assert torch.equal(ia.values, ib.values) and torch.equal(a[3], b[3].cpu())
        assert torch.allclose(a[1].gather(1, ia.indices), b[1].cpu().gather(1, ib.indices), atol=1e-5)


# ---- engine ----------------------------------------------------------------------------------------------------
TENSOR_CORES = dict(pattern="LARALR", ff="MDM", shared_weights={5: 2}, streams=3, width=96, vocab=104, heads=4, kv_heads=2, dim=32, vdim=48, rot_dims=16, chunk=50,
                    ret_heads=3, ret_dim=48, ret_vdim=80, ret_rot=32, lat_heads=4, lat_dim=24, lat_vdim=40, kv_rank=128, window=60, ff_size=136, experts=8, top=3,
                    groups=(4, 2), expert_ff=40, shared_ff=56)
GPU_CONFIGS = dict(CONFIGS, tensor_cores=TENSOR_CORES, mma_latent=dict(TENSOR_CORES, kv_rank=80, lat_heads=20, streams=4, ret_dim=64, ret_vdim=64))


@pytest.mark.parametrize("name", sorted(GPU_CONFIGS))
def test_engine_portions_against_oracle(cuda_device, name):
    cfg = small_cfg(**GPU_CONFIGS[name])
    full, w, wo = weights_for(cfg, 7)
    cuts = [50, 2, 2, 1, 1, 17, 3, 1, 40, 1]
    toks = random_tokens(cfg, sum(cuts), 5)
    want = ref_logits(full, wo, toks)
    assert rel(run_cut(make_engine(cfg, w, device="cuda", bs=16), 1, toks, cuts), want) < 3e-4
    if name == "ones":          # widths of one: a norm over one number magnifies any rounding without bound
        return
    # bf16: as close to the oracle as the same roundings on the CPU.  Every expert is chosen, since a rounding that flips a close
    # choice moves a token's output by a whole expert on either side.
    kw = dict(GPU_CONFIGS[name], groups=None)
    cfg = small_cfg(**dict(kw, top=kw.get("experts", 6)))
    full, w, wo = weights_for(cfg, 7)
    want = ref_logits(full, wo, toks).double()
    err = lambda a: float((a.double() - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt())  # noqa: E731
    bound = 0.02 + 1.5 * err(run_cut(make_engine(cfg, w, torch.bfloat16, bs=16), 1, toks, [len(toks)]))
    for bs in (16, 64):
        whole = run_cut(make_engine(cfg, w, torch.bfloat16, "cuda", bs=bs), 1, toks, [len(toks)])
        parts = run_cut(make_engine(cfg, w, torch.bfloat16, "cuda", bs=bs), 1, toks, cuts)
        assert err(whole) < bound and err(parts) < bound, (bs, bound, err(whole), err(parts))


@pytest.mark.parametrize("dt,tol", [(torch.float32, 3e-4), (torch.bfloat16, None)])
def test_mixed_batches_and_reused_slots(cuda_device, dt, tol):
    """Portions beside single tokens of others; requests end and their pages and slots go to the next: each against alone."""
    kw = GPU_CONFIGS["tensor_cores"]
    cfg = small_cfg(**(kw if tol is not None else dict(kw, groups=None, top=kw["experts"])))      # bf16: no close choices
    w = oracle.random_weights(cfg, 8)
    lens = [70, 23, 41, 9, 55]
    prompts = [random_tokens(cfg, n, n) for n in lens]
    alone = [run_cut(make_engine(cfg, w, dt, "cuda", bs=16), 1, p, [len(p)]) for p in prompts]
    eng = make_engine(cfg, w, dt, "cuda", blocks=10, bs=16, max_batch=3)
    pos, got = [0] * 5, [[] for _ in range(5)]
    waiting, live, step = list(range(5)), [], 0
    sizes = [5, 1, 30, 2, 1, 1, 12]
    while waiting or live:
        while waiting and len(live) < 3 and eng.kv.allocate(waiting[0] + 1, 1):
            live.append(waiting.pop(0))
        portions, who = [], []
        for i in list(live):
            c = min(sizes[(step + 2 * i) % len(sizes)], lens[i] - pos[i])
            if (step + i) % 5 == 4 or not eng.kv.allocate(i + 1, pos[i] + c):
                continue
            portions.append(eng.portion(i + 1, prompts[i][pos[i]:pos[i] + c], pos[i], list(range(c))))
            who.append((i, c))
            pos[i] += c
        if portions:
            lg, o = eng.forward_portions(portions).float().cpu(), 0
            for i, c in who:
                got[i].append(lg[o:o + c])
                o += c
        for i in list(live):
            if pos[i] == lens[i]:
                eng.kv.free(i + 1)
                live.remove(i)
        step += 1
        assert step < 500
    for i in range(5):
        g = torch.cat(got[i])
        if tol is not None:
            assert rel(g, alone[i]) < tol, i
        else:
            assert float((g - alone[i]).pow(2).mean().sqrt() / alone[i].pow(2).mean().sqrt()) < 0.08, i


def test_greedy_generation_with_graph_replay(cuda_device):
    """Scheduler + engine + CUDA-graph decoding in fp32 give the oracle's tokens; states of padding rows are never touched."""
    cfg = small_cfg(**GPU_CONFIGS["tensor_cores"])
    w = oracle.random_weights(cfg, 4)
    prompts = [random_tokens(cfg, n, n) for n in (5, 63, 3, 18, 49)]
    eng = make_engine(cfg, w, device="cuda", blocks=20, bs=16, max_batch=3, graphs=True)
    outs = eng.generate(prompts, max_tokens=7, temperature=0.0)
    for p, o in zip(prompts, outs):
        seq = list(p)
        for _ in range(7):
            seq.append(int(ref_logits(cfg, w, seq)[-1].argmax()))
        assert list(o) == seq[len(p):]


def test_long_decoding(cuda_device):
    cfg = small_cfg(**GPU_CONFIGS["tensor_cores"])
    w = oracle.random_weights(cfg, 12)
    toks = random_tokens(cfg, 210, 1)
    want = ref_logits(cfg, w, toks)
    assert rel(run_cut(make_engine(cfg, w, device="cuda", bs=16), 1, toks, [10] + [1] * 200), want) < 3e-4
