"""The Rapovik design in the engine against the plain implementation of tests/plain_rapovik.py.

Every test makes its own small configuration and random weights (tests/rapovik_cases.py), writes a model folder with
the engine's random-weights mode, reads it back with the plain reader, and compares logits: float32 to 2e-4 of the
largest logit, bfloat16 to 6e-2 (tiny widths average little out).  In float32 the rows of every cut must also EQUAL
the rows of the whole request bit for bit: the 32-bit kernels take a token's sums in an order that depends on its
position only.
"""
import os

import numpy as np
import pytest
import torch

import plain_rapovik as plain
from rapovik_cases import CASES, SINGLE, Harness, attention, config, dense, mamba, mlstm, moe, rel_err, write_model

pytestmark = pytest.mark.gpu
TOL = {"float32": 2e-4, "bfloat16": 6e-2}


def plain_logits(folder, tokens):
    cfg, w = plain.read_model(folder)
    return plain.forward(cfg, w, list(tokens)).numpy()


def plain_rows(folder, tokens, dtype="bfloat16"):
    """The plain logits and which rows to compare.  A token whose router's call is close (the gap between what is chosen
    and what is not below 0.01 in scores between 0 and 1) may go to another expert once the activations are rounded to bfloat16,
    and its row then differs as a whole; such rows are left out in bfloat16.  float32 keeps every row."""
    cfg, w = plain.read_model(folder)
    margins = []
    want = plain.forward(cfg, w, list(tokens), margins=margins).numpy()
    clear = np.ones(len(tokens), dtype=bool)
    if dtype != "float32":
        for per_token in margins:
            clear &= np.array(per_token) >= 0.01
    return want, clear


def err(got, want, clear=None):
    d = np.abs(got - want)
    return float((d if clear is None else d[clear]).max() / np.abs(want).max())


def close(got, want, clear, dtype):
    """float32: every row.  bfloat16: the median row and nine of ten clear rows.  The norms on the sublayers' outputs divide by the
    output's own size, and a matrix memory's read-out may cancel (a query and the few keys it holds nearly at right angles): in these tiny models the plain
    implementation's own row moves by 0.1 and more at a few tokens when what its sublayers read is rounded to bfloat16."""
    if dtype == "float32":
        return err(got, want) < TOL[dtype]
    rows = np.abs(got - want)[clear].max(axis=1) / np.abs(want).max()
    return bool((rows < TOL[dtype]).mean() >= 0.9 and np.median(rows) < 2.5e-2 and np.isfinite(got).all())


def tokens_of(rng, n, vocab):
    return rng.integers(0, vocab, n).tolist()


def _step_arrays(lengths, slots):
    """Device arrays of a step whose sequences bring ``lengths`` tokens each."""
    seq = torch.tensor([b for b, n in enumerate(lengths) for _ in range(n)], dtype=torch.int32, device="cuda")
    starts = torch.tensor(np.concatenate([[0], np.cumsum(lengths)]), dtype=torch.int32, device="cuda")
    return seq, torch.tensor(slots, dtype=torch.int32, device="cuda"), starts


# ---- each mechanism alone: kernels ----------------------------------------------------------------
def test_norms_around_a_sublayer_in_one_kernel():
    """The norm of a sublayer's output (and a bias it owes) added into the residual, and the next norm of that residual."""
    from carbon_engine_b200 import ops
    g = torch.Generator().manual_seed(1)
    for T, W in ((5, 48), (1, 36), (70, 257), (9, 512), (3, 260), (2, 4096)):
        y, x = torch.randn(T, W, generator=g) * 4, torch.randn(T, W, generator=g)
        w1, w2, bias = (torch.randn(W, generator=g) * 0.1 for _ in range(3))
        for b in (None, bias):
            for dtype in (torch.float32, torch.bfloat16, None):
                new = x.double() + plain.norm_zero_centred(y.double() + (0 if b is None else b.double()), w1.double(), 1e-5)
                nxt = plain.norm_zero_centred(new, w2.double(), 1e-3)
                xd = x.cuda()
                h = torch.zeros(T, W, dtype=dtype, device="cuda") if dtype is not None else None
                ops.rmsnorm_add_norm(y.cuda(), (1 + w1).cuda(), xd, 1e-5, None if b is None else b.cuda(), (1 + w2).cuda() if dtype else None, 1e-3, h)
                assert rel_err(xd.cpu().numpy(), new.numpy()) < 1e-6
                if dtype is not None:
                    assert rel_err(h.float().cpu().numpy(), nxt.numpy()) < (1e-6 if dtype == torch.float32 else 5e-3)


def test_clamped_gated_activation_as_the_epilogue_of_every_product_kernel():
    """min(gate + b, limit), up + b cut on both sides, g sigmoid(1.702 g) (u + 1): from the float32 kernel, the tcgen05 kernels
    (one block, persistent blocks, CTA pairs) and the library product followed by the activation's own kernel; with and
    without a bias; every clamp is reached."""
    from carbon_engine_b200 import ops, ops_tensor
    from carbon_engine_b200.parts import linear
    g = torch.Generator().manual_seed(6)
    for M, N, K in ((5, 24, 40), (8, 256, 512), (70, 136, 64), (300, 512, 128), (600, 120, 64), (1000, 384, 256), (1, 72, 200)):
        a, w = torch.randn(M, K, generator=g), torch.randn(2 * N, K, generator=g) * (2.0 / K ** 0.5)
        for bias in (None, torch.randn(2 * N, generator=g)):
            for limit in (0.7, 2.5):
                def want_of(a_, w_):
                    z = a_.double() @ w_.double().T + (0 if bias is None else bias.double().to(a_.device))
                    assert bool((z[:, :N] > limit).any()) and bool((z[:, N:] > limit).any()) and bool((z[:, N:] < -limit).any())
                    return plain.clamped_glu(z[:, :N], z[:, N:], limit).cpu().numpy()
                glu = ops.GluParams(limit, 1.702, None if bias is None else bias.cuda())
                out = torch.empty(M, N, device="cuda")
                ops.gemm_plain(a.cuda(), w.cuda(), out, ops.GEMM_CLAMPGLU, glu)
                assert rel_err(out.cpu().numpy(), want_of(a, w)) < 1e-5
                ab, wb = a.cuda().bfloat16(), w.cuda().bfloat16()
                wantb = want_of(ab, wb)
                outb = torch.full((M, N), float("nan"), device="cuda", dtype=torch.bfloat16)
                assert ops_tensor.gemm_bf16(ab, wb, outb, ops.GEMM_CLAMPGLU, glu)
                assert rel_err(outb.float().cpu().numpy(), wantb) < 1e-2
                outb.fill_(float("nan"))
                linear.BF16_BACKEND = "library"
                try:
                    linear.matmul_nt(ab, wb, outb, linear.CLAMPGLU, glu=glu)
                finally:
                    linear.BF16_BACKEND = "auto"
                assert rel_err(outb.float().cpu().numpy(), wantb) < 2e-2


def test_router_kernel_picks_what_the_plain_router_picks():
    from carbon_engine_b200 import ops
    g = torch.Generator().manual_seed(2)

    def run(z, corr, E, top, groups, keep):
        T = z.shape[0]
        ids, wts = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
        ops.moe_route(z.cuda(), E, top, groups, keep, 1.0, ids, wts, None, "sigmoid", corr.cuda(), "top2", False)
        return ids.cpu(), wts.cpu()
    for T, E, top, groups, keep in ((9, 6, 2, 3, 2), (4, 8, 4, 2, 1), (33, 5, 3, 5, 4), (7, 7, 7, 1, 1), (3, 64, 6, 8, 3), (5, 4, 1, 1, 1),
                                    (6, 12, 3, 12, 3), (2, 300, 40, 1, 1), (5, 16, 4, 4, 4)):
        z = torch.randn(T, E + 3, generator=g) * 2          # a wider row than the router needs
        corr = torch.randn(E, generator=g) * 0.7 - 0.8       # most choice scores are negative: a barred expert must not count as 0
        ids, wts = run(z, corr, E, top, groups, keep)
        router = {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}}
        for t in range(T):
            chosen, weights = plain.route(z[t, :E].double(), corr.double(), router)
            assert ids[t].tolist() == chosen, (E, top, groups, keep, t)
            assert np.allclose(wts[t].numpy(), weights, rtol=2e-6)
    # a group wins by the sum of its two largest choice scores: group 0 has the single best expert, group 1 the larger sum
    z = torch.tensor([[4.0, -9.0, -9.0, 3.0, 3.0, 3.0]])
    ids, _ = run(z, torch.zeros(6), 6, 2, 2, 1)
    assert sorted(ids[0].tolist()) == [3, 4]
    # numbers that are none leave nothing to choose: the kernel still names experts that exist
    ids, _ = run(torch.full((2, 6), float("nan")), torch.zeros(6), 6, 3, 2, 1)
    assert ((ids >= 0) & (ids < 6)).all()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gated_experts_products_over_the_layout_by_expert(dtype):
    """Route, lay out, the two grouped products (the first with the clamped gated activation of row pairs), the weighted sum and the
    shared expert, against the plain loop; tiles of 16, 64 and 128 rows; experts without a token; feature counts that are no multiple of
    the kernels' tiles; in bfloat16 the wmma kernel and the tcgen05 kernel fed by TMA as well."""
    from carbon_engine_b200 import ops, ops_tensor
    g = torch.Generator().manual_seed(3)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    for T, W, E, top, ff, sff, tile in ((13, 40, 6, 2, 12, 20, 16), (70, 48, 4, 3, 40, 16, 64), (3, 32, 16, 2, 16, 48, 16),
                                        (150, 64, 5, 1, 24, 0, 64), (1, 36, 8, 8, 7, 5, 16), (500, 136, 5, 2, 104, 0, 128)):
        rnd = lambda *s: (torch.randn(*s, generator=g) * 0.4).to(dtype).double()
        h = rnd(T, W)
        w = {"m.router": rnd(E, W) * 3, "m.correction": rnd(E)}
        for e in range(E):
            w[f"m.e{e}.gate"], w[f"m.e{e}.up"], w[f"m.e{e}.down"] = rnd(ff, W), rnd(ff, W), rnd(W, ff)
        mlp = {"router": {"experts": E, "top": top}, "expert": {"ff": ff, "limit": 0.8}}
        if sff:
            w["m.shared.gate"], w["m.shared.up"], w["m.shared.down"] = rnd(sff, W), rnd(sff, W), rnd(W, sff)
            mlp["shared"] = {"ff": sff, "limit": 1.3}
        dev = lambda t: t.to(dtype).cuda().contiguous()
        z = (h @ w["m.router"].T).float().cuda()
        ids, wts = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
        ops.moe_route(z, E, top, 1, 1, 1.0, ids, wts, None, "sigmoid", w["m.correction"].float().cuda(), "top2", False)
        want = plain.moe_ff(w, "m", mlp, h)
        tiles = ops.moe_max_tiles(T * top, E, tile)
        i32 = lambda n: torch.full((n,), -7, dtype=torch.int32, device="cuda")
        row_token, pair_row, tile_expert, n_tiles = i32(tiles * tile), i32(T * top), i32(tiles), i32(1)
        ops.moe_align(ids, E, tile, row_token, pair_row, tile_expert, n_tiles)
        up = torch.empty(E, 2 * ff, W, dtype=dtype, device="cuda")
        for e in range(E):
            up[e, 0::2], up[e, 1::2] = dev(w[f"m.e{e}.gate"]), dev(w[f"m.e{e}.up"])
        down = dev(torch.stack([w[f"m.e{e}.down"] for e in range(E)]))
        hd = dev(h)
        shared = None
        if sff:
            sact = torch.empty(T, sff, dtype=dtype, device="cuda")
            from carbon_engine_b200.parts import linear
            linear.matmul_nt(hd, dev(torch.cat([w["m.shared.gate"], w["m.shared.up"]])), sact, linear.CLAMPGLU, glu=ops.GluParams(1.3, 1.702))
            shared = torch.empty(T, W, dtype=dtype, device="cuda")
            linear.matmul_nt(sact, dev(w["m.shared.down"]), shared, linear.STORE)

        def finish(act):
            rows = torch.empty(tiles * tile, W, dtype=dtype, device="cuda")
            if tile == 128:
                assert ops_tensor.grouped_bf16(act, down, rows, tile, 0, tile_expert, n_tiles)
            else:
                ops.moe_matmul(act, down, rows, tile, "none", None, tile_expert, n_tiles)
            y = torch.full((T, W), 0.5, device="cuda")
            ops.moe_combine(rows, pair_row, wts, y, shared, None, True)
            return rel_err(y.cpu().numpy() - 0.5, want.numpy())
        if tile != 128:
            act = torch.zeros(tiles * tile, ff, dtype=dtype, device="cuda")
            ops.reset_kernel_counts()
            ops.moe_matmul(hd, up, act, tile, "clamped_glu", row_token, tile_expert, n_tiles, 0.8, 1.702)
            assert ("moe_matmul_wmma_kernel" in ops.kernel_counts()) == (dtype == torch.bfloat16 and W % 16 == 0 and ff % 8 == 0)
            assert finish(act) < tol, (T, W, E, top)
        if dtype == torch.bfloat16 and W % 8 == 0 and ff % 8 == 0:
            laid = torch.full((tiles * tile, W), float("nan"), dtype=dtype, device="cuda")
            ops.moe_gather(hd, row_token, n_tiles, tile, laid)
            act = torch.zeros(tiles * tile, ff, dtype=dtype, device="cuda")
            assert ops_tensor.grouped_bf16(laid, up, act, tile, 2, tile_expert, n_tiles, 0.8, 1.702)
            assert finish(act) < tol and ops_tensor.gemm_status(hd.device) == 0


@pytest.mark.parametrize("H, G, N, dv, K, parts", [(4, 2, 12, 8, 4, 2), (3, 3, 7, 10, 1, 5), (2, 1, 136, 8, 2, 1), (6, 2, 64, 16, 3, 6), (8, 1, 16, 128, 4, 2)])
def test_state_space_kernels(H, G, N, dv, K, parts):
    """Three sequences in three steps (portions, then single tokens, then portions again, from the state and the kept convolution
    inputs) against the walk over each whole sequence."""
    from carbon_engine_b200 import ops
    g = torch.Generator().manual_seed(H * 100 + N)
    inner, C = H * dv, 2 * G * N + H * dv
    steps = [[17, 3, 40], [1, 1, 1], [2, 33, 1]]
    ld = (C + inner + H + 3) // 4 * 4
    taps, bias = torch.randn(C, K, generator=g) * 0.5, torch.randn(C, generator=g) * 0.3
    a_log, dt_bias, skip = torch.randn(H, generator=g) * 0.5, torch.randn(H, generator=g) * 0.3, 1 + 0.5 * torch.randn(H, generator=g)
    norm_w = 1 + 0.1 * torch.randn(inner, generator=g)
    state, kept = torch.zeros(4, H, N, dv, device="cuda"), torch.zeros(4, max(K - 1, 1), C, device="cuda")
    slots = [3, 0, 2]
    rows = [torch.randn(sum(s[b] for s in steps), ld, generator=g) for b in range(3)]
    outs, at = [[], [], []], [0, 0, 0]
    ops.reset_kernel_counts()
    for lengths in steps:
        seq, slot_t, starts = _step_arrays(lengths, slots)
        T = sum(lengths)
        proj = torch.cat([rows[b][at[b]:at[b] + n] for b, n in enumerate(lengths)]).cuda()
        prep = torch.full((T, ops.gated_delta_prep_width(H, G, N, dv, ops.DECAY_PER_HEAD)), float("nan"), device="cuda")
        raw, out = torch.empty(T, inner, device="cuda"), torch.empty(T, inner, device="cuda")
        ops.gated_delta(proj, proj[:, C + inner:C + inner + H], proj[:, C:C + inner], taps.cuda(), a_log.cuda(), dt_bias.cuda(), norm_w.cuda(),
                        prep, raw, state, kept if K > 1 else None, out, seq, slot_t, starts, 3, 0, 0, H, G, N, dv, K, 1e-5,
                        decay=ops.DECAY_PER_HEAD, gate=ops.GATE_SILU, delta=False, out_scale=0.75, operands=ops.OPERANDS_CONV,
                        conv_bias=bias.cuda(), write_step=True, skip=skip.cuda(), norm_parts=parts)
        o = 0
        for b, n in enumerate(lengths):
            outs[b].append(out[o:o + n].cpu()); o += n; at[b] += n
    ran = ops.kernel_counts()
    assert ran["gated_delta_walk_kernel"] == 2 and ran["gated_delta_step_kernel"] == 1 and ran.get("gated_delta_keep_kernel", 0) == (2 if K > 1 else 0)
    for b in range(3):
        x = rows[b].double()
        n = x.shape[0]
        conv = plain.silu(plain.causal_conv(x[:, :C], taps.double(), bias.double()))
        Cm, Bm, xs = conv[:, :G * N].reshape(n, G, N), conv[:, G * N:2 * G * N].reshape(n, G, N), conv[:, 2 * G * N:].reshape(n, H, dv)
        dt = plain.softplus(x[:, C + inner:C + inner + H] + dt_bias.double())
        y = torch.stack([plain.state_space_walk(xs[:, i], Bm[:, i // (H // G)], Cm[:, i // (H // G)], dt[:, i], float(torch.exp(a_log[i].double())), float(skip[i]))
                         for i in range(H)], dim=1).reshape(n, inner)
        y = y * plain.silu(x[:, C:C + inner])
        want = plain.unit_rms(y.reshape(n, parts, inner // parts), 1e-5).reshape(n, inner) * norm_w.double() * 0.75
        assert rel_err(torch.cat(outs[b]).numpy(), want.numpy()) < 3e-5, b


@pytest.mark.parametrize("H, d, dv, cap", [(3, 8, 12, 15.0), (2, 20, 6, 1.5), (1, 136, 8, 4.0), (40, 4, 5, 8.0), (2, 64, 128, 6.0)])
def test_matrix_memory_kernels(H, d, dv, cap):
    """Gates whose logits spread far beyond the caps, so that the running maximum comes from the input gate at some tokens and from the
    decayed maximum at others, and the divisor is |n.q| at some and exp(-m) at others; portions longer than the scan's chunk, single
    tokens, and portions again."""
    from carbon_engine_b200 import ops
    g = torch.Generator().manual_seed(H * 10 + d)
    steps = [[150, 5, 64], [1, 1, 1], [3, 70, 1]]
    n_q, n_v = H * d, H * dv
    ld = (2 * n_q + 2 * n_v + 2 * H + 3) // 4 * 4
    bias, norm_w = torch.cat([torch.randn(H, generator=g), 2 + torch.randn(H, generator=g)]), 1 + 0.1 * torch.randn(n_v, generator=g)
    state, m_state = torch.zeros(4, H, d * (dv + 1), device="cuda"), torch.zeros(4, H, device="cuda")
    slots = [1, 3, 0]
    rows = [torch.randn(sum(s[b] for s in steps), ld, generator=g) for b in range(3)]
    off_g = 2 * n_q + n_v
    for r in rows:
        r[:, off_g + n_v:] *= 5.0
    outs, at = [[], [], []], [0, 0, 0]
    for lengths in steps:
        seq, slot_t, starts = _step_arrays(lengths, slots)
        T = sum(lengths)
        proj = torch.cat([rows[b][at[b]:at[b] + n] for b, n in enumerate(lengths)]).cuda()
        prep = torch.full((T, ops.gated_delta_prep_width(H, H, d, dv, ops.DECAY_EXP_GATES)), float("nan"), device="cuda")
        raw, out = torch.empty(T, H * (dv + 1), device="cuda"), torch.empty(T, n_v, device="cuda")
        ops.gated_delta(proj, proj[:, off_g + n_v:off_g + n_v + 2 * H], proj[:, off_g:off_g + n_v], None, None, bias.cuda(), norm_w.cuda(), prep, raw,
                        state, None, out, seq, slot_t, starts, 3, 0, 0, H, H, d, dv, 1, 1e-5, decay=ops.DECAY_EXP_GATES, delta=False,
                        operands=ops.OPERANDS_PLAIN, m_state=m_state, cap=cap, normalizer=True)
        o = 0
        for b, n in enumerate(lengths):
            outs[b].append(out[o:o + n].cpu()); o += n; at[b] += n
    for b in range(3):
        x = rows[b].double()
        n = x.shape[0]
        q, k, v = x[:, :n_q].reshape(n, H, d) * d ** -0.5, x[:, n_q:2 * n_q].reshape(n, H, d), x[:, 2 * n_q:off_g].reshape(n, H, dv)
        li = plain.soft_cap(x[:, off_g + n_v:off_g + n_v + H] + bias[:H].double(), cap)
        lf = plain.log_sigmoid(plain.soft_cap(x[:, off_g + n_v + H:off_g + n_v + 2 * H] + bias[H:].double(), cap))
        o = torch.stack([plain.matrix_memory_walk(q[:, i], k[:, i], v[:, i], li[:, i], lf[:, i]) for i in range(H)], dim=1)
        want = (plain.unit_rms(o, 1e-5).reshape(n, n_v) * norm_w.double() * torch.sigmoid(x[:, off_g:off_g + n_v])).numpy()
        got = torch.cat(outs[b]).numpy()
        # the read-outs n.q may cancel: what is compared is each row against its own size, nearly all rows closely
        e = np.abs(got - want).max(axis=1) / np.abs(want).max(axis=1)
        assert np.quantile(e, 0.97) < 1e-4 and e.max() < 1e-2, (b, e.max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_interleaved_rotation_in_latent_attentions_operands(dtype):
    from carbon_engine_b200 import ops
    g = torch.Generator().manual_seed(9)
    for r, dr, rd, H in ((14, 8, 8, 3), (9, 6, 4, 1), (48, 16, 16, 8), (5, 2, 2, 2)):
        T, page, base = 11, 4, 60.0
        proj = torch.randn(T, (r + dr + 3) // 4 * 4, generator=g)
        w = 1 + 0.1 * torch.randn(r, generator=g)
        pos = torch.arange(3, 3 + T, dtype=torch.int32)
        ang = torch.arange(32, dtype=torch.float64)[:, None] * torch.tensor([base ** (-2.0 * i / rd) for i in range(rd // 2)], dtype=torch.float64)[None, :]
        cos, sin = ang.cos().float().cuda(), ang.sin().float().cuda()
        pool = torch.full((5, 1, page, r + dr), float("nan"), dtype=dtype, device="cuda")
        table = torch.tensor([[-1] * 4, [4, 2, 0, 3]], dtype=torch.int32, device="cuda")
        status = torch.zeros(1, dtype=torch.int32, device="cuda")
        seq, slot = torch.zeros(T, dtype=torch.int32, device="cuda"), torch.tensor([1], dtype=torch.int32, device="cuda")
        ops.latent_prepare(proj.cuda(), None, w.cuda(), None, pool, cos, sin, pos.cuda(), seq, slot, table, status, 0, 0, 0, r, dr, rd, page, 1e-5,
                           pairing="interleaved")
        x = proj.double()
        want = torch.cat([plain.unit_rms(x[:, :r], 1e-5) * w.double(), plain.rotate_neighbours(x[:, None, r:r + dr], pos, rd, base)[:, 0]], dim=-1)
        got = torch.stack([pool[table[1, p // page], 0, p % page] for p in pos.tolist()])
        assert rel_err(got.float().cpu().numpy(), want.numpy()) < (1e-5 if dtype == torch.float32 else 1e-2)
        q = torch.randn(T, H * (3 + dr), generator=g).to(dtype)
        dst = torch.zeros(T, H * (r + dr), dtype=dtype, device="cuda")
        ops.rope_part(q.cuda(), 3 + dr, 3, dst, r + dr, r, cos, sin, pos.cuda(), status, H, dr, rd, pairing="interleaved")
        want = plain.rotate_neighbours(q.double().reshape(T, H, 3 + dr)[..., 3:], pos, rd, base)
        assert rel_err(dst.reshape(T, H, r + dr)[..., r:].float().cpu().numpy(), want.numpy()) < (1e-5 if dtype == torch.float32 else 1e-2)
        assert float(dst.reshape(T, H, r + dr)[..., :r].abs().max()) == 0.0 and int(status.item()) == 0


# ---- each mechanism alone: one layer of each kind ----------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_one_layer_of_each_kind(tmp_path, name, dtype):
    folder = write_model(SINGLE[name], str(tmp_path / name), seed=7)
    toks = tokens_of(np.random.default_rng(5), 45, SINGLE[name]["vocab"])
    want, clear = plain_rows(folder, toks, dtype)
    assert clear.sum() > 30
    h = Harness(folder, dtype)
    whole = h.run(toks)
    assert close(whole, want, clear, dtype)
    one_by_one = h.run(toks, [1])
    assert close(one_by_one, want, clear, dtype)
    if dtype == "float32":
        assert np.array_equal(whole, one_by_one)


def test_layers_outputs_one_after_another(tmp_path):
    """The residual after every layer run (a looped layer counts each time), in float32."""
    from carbon_engine_b200.engine.batch import StepEntry
    for name in ("A", "B", "C"):
        folder = write_model(CASES[name], str(tmp_path / name))
        cfg, w = plain.read_model(folder)
        toks = tokens_of(np.random.default_rng(1), 30, cfg["vocab"])
        trace = []
        plain.forward(cfg, w, toks, tap=lambda i, x: trace.append(x.clone()))
        h = Harness(folder, "float32")
        rid = h.open()
        ctx, rows, commits = h.runner.prepare([StepEntry(rid, toks, [0])])
        got = []
        h.model.forward(ctx, h.storage, tap=lambda i, x: got.append(x.clone().cpu().numpy()))
        assert len(got) == len(trace) == len(plain.layer_runs(cfg))
        for i, (a, b) in enumerate(zip(got, trace)):
            assert rel_err(a, b.numpy()) < 1e-4, (name, i)


# ---- whole models: cuts, batches, reuse ------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CASES))
def test_whole_prompt_portions_and_decoding(tmp_path, name, dtype):
    from carbon_engine_b200 import ops
    folder = write_model(CASES[name], str(tmp_path / name), seed=16)
    toks = tokens_of(np.random.default_rng(3), 140 if name in ("T", "V") else 83, CASES[name]["vocab"])
    want, clear = plain_rows(folder, toks, dtype)
    assert clear.sum() > len(toks) // 2
    h = Harness(folder, dtype, page_size=8, pages=24)          # 192 tokens of pages: every run reuses the last one's
    ops.reset_kernel_counts()
    whole = h.run(toks)
    if name in ("T", "V"):        # sizes of the tensor-core kernels: bfloat16 must have taken them, float32 never
        counts = ops.kernel_counts()
        assert ("masked_attention_mma_kernel" in counts) == (dtype == "bfloat16")
        assert ("gemm_tc_grouped_kernel" in counts) == (dtype == "bfloat16")
    assert close(whole, want, clear, dtype), "whole"
    for cuts in ([1], [2], [3, 2, 7, 2, 16, 5], [40, 1, 1, 1], [64, 19]):
        got = h.run(toks, cuts)
        assert close(got, want, clear, dtype), cuts
        if dtype == "float32":
            assert np.array_equal(got, whole), cuts
    m = h.storage.manager
    assert all(m.free_pages(g) == h.storage.groups[g].num_pages for g in range(len(h.storage.groups))) and m.free_slots() == 4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_requests_in_one_batch_with_reused_pages_and_slots(tmp_path, dtype):
    """Up to three live requests, portions beside single tokens, a request left out of some steps, finished requests'
    pages and slots taken by the next: every row equals the request alone."""
    name = "A"
    folder = write_model(CASES[name], str(tmp_path / name), seed=16)
    rng = np.random.default_rng(9)
    lengths = [61, 17, 40, 1, 2, 33, 25]
    reqs = [tokens_of(rng, n, CASES[name]["vocab"]) for n in lengths]
    want = [plain_rows(folder, t, dtype) for t in reqs]
    h = Harness(folder, dtype, page_size=8, pages=20, slots=3)          # 160 tokens: three live requests at most
    alone = [h.run(t) for t in reqs] if dtype == "float32" else None
    waiting, live, done_rows = list(range(len(reqs))), {}, {i: [] for i in range(len(reqs))}
    portions, k, step_no = [2, 5, 1, 9, 3, 14], 0, 0
    while waiting or live:
        while waiting and len(live) < 3 and sum(-(-len(reqs[i]) // 8) for i in live) + -(-len(reqs[waiting[0]]) // 8) <= 20:
            i = waiting.pop(0)
            live[i] = [h.open(), 0]
        entries, who = [], []
        for i, (rid, pos) in list(live.items()):
            if step_no % 4 == 3 and i % 2 == 0 and len(live) > 1:
                continue                                     # left out of this step
            left = len(reqs[i]) - pos
            n = 1 if left <= 6 else min(portions[k % len(portions)], left - 6)      # the last tokens one by one
            k += 1
            entries.append((rid, reqs[i][pos:pos + n], range(n)))
            who.append((i, n))
        step_no += 1
        if not entries:
            continue
        rows = h.step(entries)
        at = 0
        for i, n in who:
            done_rows[i].append(rows[at:at + n])
            at += n
            live[i][1] += n
            if live[i][1] == len(reqs[i]):
                h.close(live.pop(i)[0])
    got = [np.concatenate(done_rows[i]) for i in range(len(reqs))]
    assert close(np.concatenate(got), np.concatenate([w[0] for w in want]), np.concatenate([w[1] for w in want]), dtype)
    if alone is not None:
        for i in range(len(reqs)):
            assert np.array_equal(got[i], alone[i]), i
    assert h.storage.manager.free_slots() == 3


# ---- a key that stands out: far away, at page borders, at a window's edges ------------------------------------------------
def standout_model(tmp_path, tag, window=None, heads=2, dim=16, rot_dim=16, vdim=16, kv_rank=32):
    """One latent-attention layer in which EVERY query scores the marker token's key far above hundreds of others: the first
    embedding element is the same large number for every token, one unrotated query element reads it, and one element of the
    cached latent reads an embedding element that only the marker has.  The output takes one direction from that latent element and
    another from a latent element that all tokens share (the norm on the mixer's output would undo a mere change of length)."""
    W = 32
    raw = config([attention(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=1.0, base=1e4, window=window)], width=W, vocab=50)

    def change(t):
        dt = t["embed"].dtype
        e = t["embed"].float() * 30.0
        e[:, 0], e[:, 1] = 3.0, 0.0
        e[7, 1] = 3.0
        t["embed"] = e.to(dt)
        t["l0.norm1"] = torch.zeros(W)
        dkv, q, uk, uv, o = (t[f"l0.mix.{n}"].float() for n in ("dkv", "q", "uk", "uv", "o"))
        dkv[3], dkv[4] = 0.0, 0.0
        dkv[3, 1], dkv[4, 0] = 1.0, 2.0
        t["l0.mix.dkv.norm"] = torch.ones(kv_rank)
        sign = lambda k: torch.tensor([1.0 if (k * c) % 7 < 4 else -1.0 for c in range(W)])
        for i in range(heads):
            row = i * (dim + rot_dim) + 2
            q[row] = 0.0
            q[row, 0] = 1.6
            uk[i * dim + 2], uv[i * vdim + 1], uv[i * vdim + 2] = 0.0, 0.0, 0.0
            uk[i * dim + 2, 3], uv[i * vdim + 1, 3], uv[i * vdim + 2, 4] = 2.0, 1.0, 0.1
            o[:, i * vdim + 1], o[:, i * vdim + 2] = (0.5 + 0.3 * i) * sign(3), sign(5)
        for n, v in (("dkv", dkv), ("q", q), ("uk", uk), ("uv", uv), ("o", o)):
            t[f"l0.mix.{n}"] = v.to(dt)
    return write_model(raw, str(tmp_path / f"standout_{tag}"), seed=21, change=change)


def marker_effect(folder, toks, at):
    """How far the plain model's rows move when the marker at ``at`` is replaced by an ordinary token."""
    want = plain_logits(folder, toks)
    other = list(toks)
    other[at] = 9
    return want, np.abs(want - plain_logits(folder, other)).max(axis=1) / np.abs(want).max()


@pytest.mark.parametrize("sizes", [dict(dim=6, rot_dim=4, vdim=6, kv_rank=9), dict(heads=8)])      # the float32-arithmetic kernel; the tensor-core kernel
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_key_among_hundreds_and_at_page_borders(tmp_path, dtype, sizes):
    from carbon_engine_b200 import ops
    folder = standout_model(tmp_path, "far", **sizes)
    rng = np.random.default_rng(6)
    base = [int(t) for t in rng.integers(10, 50, 720)]
    h = Harness(folder, dtype, page_size=16, pages=48, max_step_tokens=1024)
    ops.reset_kernel_counts()
    for marker_at in (3, 15, 16):
        toks = list(base)
        toks[marker_at] = 7
        want, moved = marker_effect(folder, toks, marker_at)
        assert moved[marker_at:].min() > 0.1 and moved[:marker_at].max(initial=0.0) < 1e-12          # the plain model says the far key matters
        assert rel_err(h.run(toks), want) < TOL[dtype], marker_at
        rid = h.open()
        rows = [h.step([(rid, toks[:690], [689])])]
        for p in range(690, 720):
            rows.append(h.step([(rid, toks[p:p + 1], [0])]))
        h.close(rid)
        assert rel_err(np.concatenate(rows), want[689:]) < TOL[dtype], marker_at
    assert ("masked_attention_mma_kernel" in ops.kernel_counts()) == (dtype == "bfloat16" and "heads" in sizes)


@pytest.mark.parametrize("window", [1, 2, 16, 37, 64, 65, 130])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_key_just_inside_and_just_outside_the_window(tmp_path, dtype, window):
    """The row window - 1 tokens after the marker still sees it, the next one does not; in whole prompts, in portions cut around the
    edge and in decoding, with pages given back as the window passes, and with the tensor-core kernel's sizes."""
    folder = standout_model(tmp_path, f"w{window}", window=window, heads=8)
    rng = np.random.default_rng(window)
    h = Harness(folder, dtype, page_size=8, pages=40)
    for marker_at in (0, 7, 8, 21):
        n = marker_at + window + 6
        toks = [int(t) for t in rng.integers(10, 50, n)]
        toks[marker_at] = 7
        want, moved = marker_effect(folder, toks, marker_at)
        inside, outside = marker_at + window - 1, marker_at + window
        assert moved[marker_at:outside].min() > 0.1 and moved[outside:].max() < 1e-12
        whole = h.run(toks)
        assert rel_err(whole, want) < TOL[dtype], (marker_at, "whole")
        for cuts in ([1], [2], [max(1, inside), 1], [max(1, outside), 2], [marker_at + 1, 3]):
            got = h.run(toks, cuts)
            assert rel_err(got, want) < TOL[dtype], (marker_at, cuts)
            if dtype == "float32":
                assert np.array_equal(got, whole)


# ---- the states -----------------------------------------------------------------------------------------------------------
def test_long_decoding_keeps_the_state(tmp_path):
    """300 tokens one by one after a short prompt, in float32: the recurrent states, the running maxima, the convolutions' kept rows
    and the pages must carry every token (bit for bit the rows of the whole prompt)."""
    folder = write_model(CASES["C"], str(tmp_path / "C"), seed=2)
    toks = tokens_of(np.random.default_rng(8), 310, CASES["C"]["vocab"])
    want = plain_logits(folder, toks)
    h = Harness(folder, "float32", page_size=8, pages=48)
    whole = h.run(toks)
    got = h.run(toks, [10] + [1] * 300)
    assert rel_err(got, want) < TOL["float32"] and np.array_equal(got, whole)


def test_an_early_token_reaches_far_through_the_states(tmp_path):
    """With step sizes and forget gates that hardly decay a token still counts 400 tokens later, in the state-space mixer and in
    the matrix memory: the plain model says so, and the engine's decoded rows agree with it."""
    for kind in ("mamba", "mlstm"):
        layer = mamba(heads=2, vdim=8, state=12, groups=1, conv=2, norm_groups=1) if kind == "mamba" else mlstm(heads=2, dim=12, vdim=8)

        def change(t):
            if kind == "mamba":
                t["l0.mix.A_log"] = torch.tensor([-7.0, -8.0])
            else:
                t["l0.mix.f.b"] = torch.tensor([9.0, 8.0])
                t["l0.mix.f"] = t["l0.mix.f"] * 0.1
        raw = config([layer])
        folder = write_model(raw, str(tmp_path / kind), seed=4, change=change)
        toks = tokens_of(np.random.default_rng(10), 420, raw["vocab"])
        want, moved = marker_effect(folder, toks, 2)
        assert moved[400:].min() > 5e-4, kind
        h = Harness(folder, "float32", page_size=8, pages=60, max_step_tokens=512)
        rid = h.open()
        rows = [h.step([(rid, toks[:395], [394])])] + [h.step([(rid, toks[p:p + 1], [0])]) for p in range(395, 420)]
        h.close(rid)
        assert rel_err(np.concatenate(rows), want[394:]) < 0.1 * moved[400:].min(), kind


def test_gates_beyond_their_caps_and_large_step_sizes(tmp_path):
    """Biases that push the input gates far up and down, the forget gates to their bound and the step sizes to where softplus is
    linear: the caps, the running maximum and the divisor's other branch show in the logits (the plain model without them differs)."""
    raw = config([mlstm(heads=3, gate_cap=5.0), mamba()])

    def change(t):
        t["l0.mix.i.b"] = torch.tensor([9.0, -9.0, 0.5])
        t["l0.mix.f.b"] = torch.tensor([1.0, 7.0, -4.0])
        t["l1.mix.dt_bias"] = torch.tensor([25.0, -6.0, 3.0, 0.0])
    folder = write_model(raw, str(tmp_path / "m"), seed=6, change=change)
    toks = tokens_of(np.random.default_rng(4), 120, raw["vocab"])
    want = plain_logits(folder, toks)
    other = dict(raw, layers=[mlstm(heads=3, gate_cap=50.0), raw["layers"][1]])
    cfg, w = plain.read_model(folder)
    assert rel_err(plain.forward(other, w, toks).numpy(), want) > 1e-2
    for dtype in ("float32", "bfloat16"):
        h = Harness(folder, dtype)
        for cuts in (None, [1], [70, 2, 1]):
            assert rel_err(h.run(toks, cuts), want) < TOL[dtype], (dtype, cuts)


def test_first_tokens_of_a_sequence_in_a_reused_slot(tmp_path):
    """A slot and pages that held a longer request: the next request's first tokens must start from nothing (zero
    states and maxima, no kept convolution inputs, no keys), also when it is shorter than the convolution."""
    for name in ("A", "C"):
        folder = write_model(CASES[name], str(tmp_path / name), seed=5)
        rng = np.random.default_rng(12)
        h = Harness(folder, "float32", page_size=8, pages=12, slots=1, poison=False)
        h.run(tokens_of(rng, 90, CASES[name]["vocab"]))
        for n in (1, 2, 3, 9):
            toks = tokens_of(rng, n, CASES[name]["vocab"])
            want = plain_logits(folder, toks)
            assert rel_err(h.run(toks), want) < TOL["float32"]
            assert rel_err(h.run(toks, [1]), want) < TOL["float32"]


# ---- through the entry point -------------------------------------------------------------------------
@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_engine(tmp_path, graphs):
    from carbon_engine_b200 import Engine, SamplingParams
    folder = write_model(CASES["A"], str(tmp_path / "A"), seed=17)
    cfg, w = plain.read_model(folder)
    rng = np.random.default_rng(2)
    prompts = [tokens_of(rng, n, cfg["vocab"]) for n in (23, 5, 41)]
    eng = Engine(folder, dtype="float32", page_size=8, max_running_requests=3, max_prefill_tokens=16, kv_tokens=256,
                 cuda_graphs=graphs)
    assert eng.cuda_graphs == graphs
    outs = eng.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True))
    for prompt, out in zip(prompts, outs):
        assert len(out.token_ids) == 12 and out.finish_reason == "length"
        toks = list(prompt)
        for t in out.token_ids:
            row = plain.forward(cfg, w, toks)[-1]
            assert t == int(row.argmax()) or float(row.max() - row[t]) < 4e-4 * float(row.abs().max())
            toks.append(t)
    eng.storage.manager.check()


def test_trace_replay_program_on_a_rapovik_folder(tmp_path):
    import json, subprocess, sys
    from helpers import ROOT
    folder = write_model(CASES["B"], str(tmp_path / "B"), seed=1)
    toks = tokens_of(np.random.default_rng(3), 40, CASES["B"]["vocab"])
    want = plain_logits(folder, toks)
    out = str(tmp_path / "out")
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:25], "want": [0, 24]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[25:27], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[27:], "want": [12]}, {"id": "b", "tokens": toks[:3], "want": [2]}],
              "end": ["a", "b"]}]
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32",
                           "--out", out, "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    got0 = np.fromfile(os.path.join(out, "0.f32"), dtype="<f4").reshape(2, -1)
    got2 = np.fromfile(os.path.join(out, "2.f32"), dtype="<f4").reshape(2, -1)
    assert not os.path.exists(os.path.join(out, "1.f32"))
    assert rel_err(got0, want[[0, 24]]) < 2e-4 and rel_err(got2, want[[39, 2]]) < 2e-4


def test_command_line_writes_and_generates_a_rapovik_model(tmp_path):
    """``tiny-model --arch rapovik`` then ``generate``: the printed ids are the plain implementation's greedy ones."""
    import ast, re, subprocess, sys
    from helpers import ROOT
    carbon = [sys.executable, os.path.join(ROOT, "bin", "carbon")]
    out = str(tmp_path / "tiny_r")
    p = subprocess.run(carbon + ["tiny-model", "--arch", "rapovik", "--out", out, "--layers", "4", "--hidden", "48", "--heads", "3",
                                 "--head-dim", "16", "--vocab", "120", "--seed", "9", "--loop", "1,3,2", "--mask-size", "12", "--experts", "6",
                                 "--expert-groups", "3", "--max-positions", "256"], capture_output=True, text=True, timeout=600)
    assert p.returncode == 0 and "wrote" in p.stdout, p.stderr[-2000:]
    cfg, w = plain.read_model(out)
    assert cfg["architecture"] == "Rapovik" and len(cfg["layers"]) == 4 and cfg["loop"] == {"start": 1, "stop": 3, "times": 2}
    prompt = tokens_of(np.random.default_rng(5), 17, 120)
    p = subprocess.run(carbon + ["generate", "--model", out, "--prompt-ids", ",".join(map(str, prompt)), "--max-tokens", "8",
                                 "--ignore-eos", "--print-ids", "--dtype", "f32", "--kv-tokens", "256", "--page-size", "16"],
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    ids = [ast.literal_eval(m) for m in re.findall(r"output_ids: (\[[^\]]*\])", p.stderr)][0]
    toks = list(prompt)
    for t in ids:
        row = plain.forward(cfg, w, toks)[-1]
        assert t == int(row.argmax()) or float(row.max() - row[t]) < 4e-4 * float(row.abs().max())
        toks.append(t)
    assert len(ids) == 8
