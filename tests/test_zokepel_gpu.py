"""Zokepel's CUDA kernels against the CPU restatements of the same ops and the engine on a GPU against the plain oracle
(``zokepel_oracle.py``), in fp32 (tight) and bf16 (rounding-sized)."""
import pytest
import torch

import zokepel_oracle as oracle
from test_zokepel_cpu import CONFIGS, make_engine, paged, random_tokens, ref_logits, run_cut, small_cfg

pytestmark = pytest.mark.gpu


def rel(a, b):
    """Largest row error: rms of the difference (mean taken off) over the rms of the reference row."""
    d = a.double().cpu() - b.double().cpu()
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / b.double().cpu().pow(2).mean(-1).sqrt().clamp_min(1e-9)).max())


@pytest.mark.parametrize("T,W", [(5, 10), (33, 37), (7, 320), (3, 2048), (2, 5000), (2, 9000)])
def test_glue_kernels(cuda_device, T, W):
    """Residual update with one output or a branch sum, rejoining rows, zero to two norms; the embedding."""
    from llmctl_b200.ops import dual_norm as D
    torch.manual_seed(W)
    x, e = torch.randn(T, W) * 2, torch.randn(T, W)
    ws = [torch.rand(W) + 0.5 for _ in range(4)]
    g = lambda t: None if t is None else t.to(cuda_device)  # noqa: E731
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 4e-2)):
        a, b, f = (torch.randn(T, W + 8).to(dt)[:, :W] * s for s in (0.2, 4.0, 1.0))
        a2 = torch.randn(T, 2 * W + 4).to(dt)[:, W + 4:]        # a strided view
        for pair, m, ff, add, S in ((True, a, f, e, 2), (False, a2, f, None, 2), (False, a, None, e, 1), (True, a2, None, None, 0), (False, None, None, None, 2)):
            mc = D.BranchSum(m, b, ws[0], ws[1], 0.5) if pair else m
            mg = D.BranchSum(g(m), g(b), g(ws[0]), g(ws[1]), 0.5) if pair else g(m)
            xc, xg = x.clone(), g(x.clone())
            hc = D.residual_dual_norm(mc, ff, xc, 1e-4, ws[2:2 + S], dt, add=add)
            hg = D.residual_dual_norm(mg, g(ff), xg, 1e-4, [g(w) for w in ws[2:2 + S]], dt, add=g(add))
            assert torch.allclose(xg.cpu(), xc, atol=2e-5, rtol=1e-5) and len(hg) == S
            for u, v in zip(hg, hc):
                assert u.dtype == dt and torch.allclose(u.float().cpu(), v.float(), atol=tol, rtol=1e-2)
        table = torch.randn(11, W).to(dt)
        toks, pos = torch.randint(0, 11, (T,)), torch.randint(0, 200000, (T,), dtype=torch.int32)
        fr = D.sinusoid_frequencies(W)
        xc, _ = D.embed_sinusoid(toks, pos, table, 1.7, fr)
        xg, cg = D.embed_sinusoid(g(toks), g(pos), g(table), 1.7, g(fr), want_copy=True)
        assert torch.allclose(xg.cpu(), xc, atol=2e-6) and torch.equal(xg, cg)


def test_tanh_and_head_norm_kernels(cuda_device):
    from llmctl_b200.ops import elementwise as E
    from llmctl_b200.ops import recurrent as R
    torch.manual_seed(0)
    for dt, tol in ((torch.float32, 1e-6), (torch.bfloat16, 1e-2)):
        z = torch.randn(9, 40).to(dt) * 3
        zg = z.clone().to(cuda_device)
        E.tanh_(zg[:, 3:20])
        E.tanh_(z[:, 3:20])
        assert torch.allclose(zg.float().cpu(), z.float(), atol=tol)
        H, e = 3, 21
        o, gate = torch.randn(8, H * e) * 2, torch.randn(8, H * e + 5).to(dt)[:, 5:]
        for w in (torch.rand(e) + 0.5, torch.rand(H * e) + 0.5):
            for act in ("silu", "sigmoid"):
                want = R.gla_output(o, w, gate, H, e, 1e-4, dt, act)
                got = R.gla_output(o.to(cuda_device), w.to(cuda_device), gate.to(cuda_device), H, e, 1e-4, dt, act)
                assert torch.allclose(got.float().cpu(), want.float(), atol=10 * tol, rtol=1e-2)


def portions_of(lens, pos, slots, device="cpu"):
    starts = [sum(lens[:i]) for i in range(len(lens))]
    p = torch.tensor([[starts[i], lens[i], pos[i], slots[i]] for i in range(len(lens))], dtype=torch.int32)
    rows = torch.tensor(sum(([i] * n for i, n in enumerate(lens)), []), dtype=torch.int32)
    return p.to(device), rows.to(device)


# sizes on every padded row count (32, 64, 128, 256) and beside it, odd and vector-aligned value sizes, several column blocks
SIZES = [(4, 2, 6, 10, 3), (2, 2, 32, 32, 4), (6, 3, 40, 36, 2), (4, 1, 64, 100, 1), (2, 1, 128, 128, 4), (3, 3, 97, 33, 6), (2, 2, 256, 64, 3),
         (1, 1, 1, 1, 4), (2, 1, 200, 260, 4)]


@pytest.mark.parametrize("H,G,d,e,taps", SIZES)
@pytest.mark.parametrize("per_channel", [False, True])
def test_delta_rule_kernels(cuda_device, H, G, d, e, taps, per_channel):
    """Prepare + scan + head norm for portions of unequal lengths side by side (one without a slot, one at position 0 over
    garbage), then decoding steps by the single-launch kernel, all from the same evolving states."""
    from llmctl_b200.ops import matrix_state as M
    torch.manual_seed(H * d + e)
    dev = cuda_device
    C, nz = 2 * G * d + H * e, H * d if per_channel else H
    conv_w, dtb, speed, nw = torch.randn(C, taps), torch.rand(nz) * 4 - 5, torch.exp(torch.rand(H) * 2 - 1.5), torch.rand(e) + 0.5
    for dt, tol in ((torch.float32, 3e-5), (torch.bfloat16, 2e-2)):
        st, cv = torch.randn(4, H, d, e), torch.randn(4, taps - 1, C)
        if dt == torch.bfloat16:
            cv = cv.to(dt).float()
        sg, cg = st.clone().to(dev), cv.clone().to(dev)
        pos, slots = [5, 0, 9], [2, 0, -1]
        for lens in ([19, 37, 3], [2, 1, 16], [1, 1, 1], [1, 1, 1], [33, 1, 2], [1, 1, 1]):
            T = sum(lens)
            p = torch.randn(T, C + nz + H + H * e + 3).to(dt)
            cut = [0, C, C + nz, C + nz + H, C + nz + H + H * e]
            po, ro = portions_of(lens, pos, slots)
            decode = max(lens) == 1

            def run(p, po, ro, st, cv, dev):
                v = [p[:, cut[i]:cut[i + 1]] for i in range(4)]
                return M.delta_rule(v[0], conv_w.to(dev), v[1], dtb.to(dev), speed.to(dev), v[2], v[3], nw.to(dev), po.to(dev), ro.to(dev), st, cv,
                                    H, G, d, e, per_channel, 1e-5, "sigmoid" if per_channel else "silu", decode=decode)
            want = run(p, po, ro, st, cv, "cpu")
            got = run(p.to(dev), po, ro, sg, cg, dev)
            assert got.dtype == dt and torch.allclose(got.float().cpu(), want.float(), atol=tol * max(1.0, float(want.float().abs().max())), rtol=0)
            assert torch.allclose(sg.cpu(), st, atol=2e-5 * max(1.0, float(st.abs().max()))) and torch.equal(cg.cpu(), cv)
            pos = [a + b for a, b in zip(pos, lens)]


@pytest.mark.parametrize("H,d", [(3, 5), (2, 32), (4, 64), (2, 100), (1, 128), (2, 256), (1, 1)])
def test_bonus_memory_kernels(cuda_device, H, d):
    """Token shift, prepare + scan and the single-launch decoding step, as above; widths on the vector and the scalar path.  (eps
    is large because a first token's output is its bonus sum times v: where that sum nearly cancels, the head norm would
    magnify the rounding of either side.)"""
    from llmctl_b200.ops import matrix_state as M
    torch.manual_seed(H + d)
    dev = cuda_device
    n = H * d
    w0, u, nw = torch.rand(n) * 6 - 6, torch.randn(n), torch.rand(n) + 0.5
    for W in (12, 31):
        mu = torch.rand(5, W)
        for dt, tol in ((torch.float32, 3e-5), (torch.bfloat16, 2e-2)):
            st, sh = torch.randn(4, H, d, d), torch.randn(4, W).to(dt).float()
            sg, hg = st.clone().to(dev), sh.clone().to(dev)
            pos, slots = [5, 0, 9], [2, 0, -1]
            for lens in ([19, 37, 3], [2, 1, 16], [1, 1, 1], [1, 1, 1], [33, 1, 2]):
                T = sum(lens)
                h, p = torch.randn(T, W).to(dt), torch.randn(T, 5 * n + 3).to(dt)
                po, ro = portions_of(lens, pos, slots)

                def run(h, p, po, ro, st, sh, dev):
                    mix = M.token_shift(h, mu.to(dev), po.to(dev), ro.to(dev), sh)
                    r, k, v, z, g = (p[:, i * n:(i + 1) * n] for i in range(5))
                    return mix, M.bonus_memory(r, k, v, z, w0.to(dev), u.to(dev), g, nw.to(dev), h, po.to(dev), st, sh, H, d, 1e-2,
                                               decode=max(lens) == 1)
                mc, want = run(h, p, po, ro, st, sh, "cpu")
                mg, got = run(h.to(dev), p.to(dev), po, ro, sg, hg, dev)
                assert torch.allclose(mg.float().cpu(), mc.float(), atol=1e-6 if dt == torch.float32 else 2e-2)
                assert torch.allclose(got.float().cpu(), want.float(), atol=tol * max(1.0, float(want.float().abs().max())), rtol=0)
                assert torch.allclose(sg.cpu(), st, atol=2e-5 * max(1.0, float(st.abs().max()))) and torch.equal(hg.cpu(), sh)
                pos = [a + b for a, b in zip(pos, lens)]


@pytest.mark.parametrize("H,G,d,e,n,bs,rows,far", [(4, 2, 8, 6, 45, 16, 8, 30.0), (3, 1, 5, 7, 133, 16, 4, 9.0), (8, 2, 16, 16, 300, 64, 16, 200.0),
                                                   (8, 4, 48, 40, 200, 64, 12, 17.5), (4, 4, 32, 64, 150, 8, 2, 3.0), (16, 2, 128, 128, 290, 64, 32, 128.0),
                                                   (2, 1, 16, 136, 70, 16, 8, 64.0), (6, 6, 64, 72, 400, 64, 10, 600.0),
                                                   (2, 1, 64, 16, 140, 64, 6, 50.0)])      # shared memory exactly at the default limit
def test_biased_attention_kernels(cuda_device, H, G, d, e, n, bs, rows, far):
    """Unit-RMS queries and keys with temperature, cache append and attention with a bias table on the FMA and tensor-core
    kernels: prompt tiles, single tokens, key slices; a prompt and a later portion of it."""
    from llmctl_b200.ops import softcap_attention as S
    dev = cuda_device
    torch.manual_seed(H * d)
    proj = torch.randn(n, H * d + G * d + G * e)
    table = S.bucket_bias_table(torch.randn(rows, H) * 2, far)
    bc, pages = paged(n, bs, seed=n)
    bg, _ = paged(n, bs, device=dev, seed=n)
    scale = 1.0 / d ** 0.5
    for dt, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
        pc = proj.to(dt)
        cc = torch.zeros(len(pages) + 3, bs, G * (d + e), dtype=dt)
        cg = torch.zeros_like(cc, device=dev)
        qc = S.window_kv_append(pc, None, H, G, d, e, False, 1e-4, bc.slots, cc, qk_norm=True, q_temp=(0.5, 32), positions=bc.positions)
        qg = S.window_kv_append(pc.to(dev), None, H, G, d, e, False, 1e-4, bg.slots, cg, qk_norm=True, q_temp=(0.5, 32), positions=bg.positions)
        assert torch.allclose(qg.cpu(), qc, atol=1e-5) and torch.allclose(cg.float().cpu(), cc.float(), atol=1e-5 if dt == torch.float32 else 3e-2)
        cg.copy_(cc)                            # the same keys on both sides: a rounding flip must not count against the attention
        want = None
        for width, splits, mma in ((16, 0, False), (1, 1, False), (1, 3, False), (128, 0, True), (1, 1, True), (1, 4, True)):
            if mma and not S.uses_tensor_cores(dt, H, G, d, e, width):
                continue
            for first in (0, n // 3):
                tiles = torch.tensor([[s, min(width, n - s), 0, 0] for s in range(first, n, width)], dtype=torch.int32)
                args = (None, None, None, scale, 0.0, 0, 0, H, G, d, e, bs, dt)
                if want is None:
                    t16 = torch.tensor([[s, min(16, n - s), 0, 0] for s in range(0, n, 16)], dtype=torch.int32)
                    want = S.softcap_window_attention(qc, cc, bc.block_tables, t16, 16, bc.positions, *args, table=table)
                got = S.softcap_window_attention(qg, cg, bg.block_tables, tiles.to(dev), width, bg.positions, *args, max_context=n, splits=splits,
                                                 tensor_cores=mma, table=table.to(dev))
                assert torch.allclose(got.float().cpu()[first:], want.float()[first:], atol=tol, rtol=1e-2), (dt, width, splits, mma, first)


@pytest.mark.parametrize("d,e", [(16, 8), (6, 5)])
def test_bias_bucket_edges_decide(cuda_device, d, e):
    """Zero scores and one dominant bucket: the output is the mean value of exactly the keys in it (fp32 and bf16 kernels)."""
    from llmctl_b200.ops import softcap_attention as S
    dev, n, bs, rows, far = cuda_device, 300, 16, 10, 180.0
    torch.manual_seed(d)
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        v = torch.randn(n, e).to(dt)
        batch, pages = paged(n, bs, device=dev, seed=3)
        cache = torch.zeros(len(pages) + 3, bs, d + e, dtype=dt, device=dev)
        proj = torch.cat([torch.zeros(n, 2 * d, dtype=dt), v], -1).to(dev)
        qo = S.window_kv_append(proj, None, 1, 1, d, e, False, 1e-6, batch.slots, cache, qk_norm=True)
        for star in range(rows):
            relb = torch.zeros(rows, 1)
            relb[star] = 40.0
            table = S.bucket_bias_table(relb, far).to(dev)
            member = torch.tensor([oracle.bucket(x, rows, far) == star for x in range(n)])
            dist = torch.arange(n)[:, None] - torch.arange(n)[None, :]
            seen = (dist >= 0) & member[dist.clamp_min(0)]
            none = ~seen.any(-1, keepdim=True)
            wgt = torch.where(none, dist >= 0, seen).double()
            want = (wgt / wgt.sum(-1, keepdim=True)) @ v.double()
            for width in (1, 16, 128):
                if width == 128 and not S.uses_tensor_cores(dt, 1, 1, d, e, width):
                    continue
                tiles = torch.tensor([[s, min(width, n - s), 0, 0] for s in range(0, n, width)], dtype=torch.int32, device=dev)
                out = S.softcap_window_attention(qo, cache, batch.block_tables, tiles, width, batch.positions, None, None, None, 1.0, 0.0, 0, 0, 1, 1,
                                                 d, e, bs, dt, max_context=n, table=table)
                assert torch.allclose(out.double().cpu(), want, atol=tol), (dt, star, width)


# ---- engine ----------------------------------------------------------------------------------------------------
GPU_CONFIGS = dict(CONFIGS, tensor_cores=dict(pattern="CPDP", ff="1111", loop=(1, 4, 2), width=96, vocab=104, heads=4, kv_heads=2, dim=24, vdim=40,
                                              conv=4, decay_rank=12, gate_rank=20, att_heads=4, att_kv_heads=2, att_dim=32, att_vdim=48,
                                              bias_rows=14, bias_max=100.0, q_temp=(0.3, 50), mix_heads=2, mix_dim=48, mix_rank=20, ff_size=136))


@pytest.mark.parametrize("name", sorted(GPU_CONFIGS))
def test_engine_portions_against_oracle(cuda_device, name):
    cfg = small_cfg(**GPU_CONFIGS[name])
    w = oracle.random_weights(cfg, 7)
    cuts = [50, 2, 2, 1, 1, 17, 3, 1, 40, 1]
    toks = random_tokens(cfg, sum(cuts), 5)
    want = ref_logits(cfg, w, toks)
    got = run_cut(make_engine(cfg, w, device="cuda", bs=16), 1, toks, cuts)
    assert rel(got, want) < 2e-4
    whole = run_cut(make_engine(cfg, w, torch.bfloat16, "cuda", bs=16), 1, toks, [len(toks)])
    parts = run_cut(make_engine(cfg, w, torch.bfloat16, "cuda", bs=16), 1, toks, cuts)
    err = lambda a: float((a.double() - want.double()).pow(2).mean().sqrt() / want.double().pow(2).mean().sqrt())  # noqa: E731
    assert err(whole) < 0.06 and err(parts) < 0.06


@pytest.mark.parametrize("dt,tol", [(torch.float32, 2e-4), (torch.bfloat16, None)])
def test_mixed_batches_and_reused_slots(cuda_device, dt, tol):
    """Portions beside single tokens of others; requests end and their pages and slots go to the next: each against alone."""
    cfg = small_cfg(**GPU_CONFIGS["tensor_cores"])
    w = oracle.random_weights(cfg, 8)
    lens = [70, 23, 41, 9, 55]
    prompts = [random_tokens(cfg, n, n) for n in lens]
    alone = []
    for p in prompts:
        alone.append(run_cut(make_engine(cfg, w, dt, "cuda", bs=16), 1, p, [len(p)]))
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
            assert float((g - alone[i]).pow(2).mean().sqrt() / alone[i].pow(2).mean().sqrt()) < 0.06, i


def test_greedy_generation_with_graph_replay(cuda_device):
    """Scheduler + engine + CUDA-graph decoding in fp32 give the oracle's tokens; states of padding rows are never touched."""
    cfg = small_cfg(**GPU_CONFIGS["tensor_cores"])
    w = oracle.random_weights(cfg, 4)
    prompts = [random_tokens(cfg, n, n) for n in (5, 33, 3, 18, 7)]
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
    assert rel(run_cut(make_engine(cfg, w, device="cuda", bs=16), 1, toks, [10] + [1] * 200), want) < 2e-4
