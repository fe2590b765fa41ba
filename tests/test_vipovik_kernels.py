"""Each mechanism of Vipovik through its kernels alone, against the plain implementation (GPU)."""
import numpy as np
import pytest
import torch

import plain_vipovik as pv
from test_fororax_attention import _paged
from test_fororax_kernels import DTYPES, dev, rounded

pytestmark = pytest.mark.gpu


def ints(*v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_rotation_then_a_norm_per_head(dtype):
    """All of a head rotated, part of it, none; widths in and out of steps of four and up to the limit; positions far out;
    columns behind q and k left alone; with and without weights."""
    from cbis_b200.kernels import ops
    g = torch.Generator().manual_seed(1)
    for T, H, G, D, dims, extra in ((5, 4, 2, 16, 16, 8), (33, 3, 1, 20, 12, 3), (7, 2, 2, 9, 6, 3), (3, 5, 0, 130, 64, 0), (2, 2, 1, 512, 512, 4),
                                    (200, 8, 2, 128, 128, 0), (9, 3, 3, 64, 32, 4), (4, 2, 1, 10, 0, 2), (6, 1, 1, 511, 2, 1)):
        rot = {"base": 700.0, "dims": dims, "scaling": {"factor": 5.0, "original": 80, "fast": 9.0, "slow": 0.6}} if dims else None
        n = (H + G) * D
        x = rounded(torch.randn(T, n + extra, generator=g) * 2, dtype)
        pos = torch.randint(0, 3000, (T,), generator=g)
        f, length = pv.frequencies(rot) if dims else (np.zeros(0), 1.0)
        freqs = torch.from_numpy(f).float().cuda() if dims else None
        # the angle is a 32-bit product of the position and the 32-bit frequency, in both
        a = (pos.float()[:, None] * torch.from_numpy(f).float()[None]).double().numpy()
        heads = x[:, :n].numpy().reshape(T, H + G, D).copy()
        u, v = heads[..., :dims // 2].copy(), heads[..., dims // 2:dims].copy()
        c, s = np.cos(a)[:, None] * length, np.sin(a)[:, None] * length
        heads[..., :dims // 2], heads[..., dims // 2:dims] = u * c - v * s, v * c + u * s
        wq, wk = 1 + 0.3 * torch.randn(D, generator=g), 1 + 0.3 * torch.randn(D, generator=g)
        for weights in (False, True):
            buf = dev(x.float(), dtype)
            ops.qk_turn_norm(buf, 0, H, H * D, G, D, 1e-3, pos.int().cuda(), freqs, dims, length, *((wq.cuda(), wk.cuda()) if weights else ()))
            ref = np.concatenate([pv.rms_norm(heads[:, :H], wq.numpy() if weights else None, 1e-3),
                                  pv.rms_norm(heads[:, H:], wk.numpy() if weights else None, 1e-3)], 1).reshape(T, n)
            got = buf.double().cpu().numpy()
            assert np.abs(got[:, :n] - ref).max() < (2e-5 if dtype == "float32" else 3e-2), (T, H, G, D, dims)
            assert np.array_equal(got[:, n:], x[:, n:].numpy())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_blends_with_the_row_before(dtype):
    """Segments of one row, of two, and longer than a block walks, over several steps with slots used again: the row before a
    segment's first one is the last of its request's step before; padding rows come out as zeros and change nothing."""
    from cbis_b200.kernels import ops
    g = torch.Generator().manual_seed(2)
    for W, n_mix, pad in ((24, 5, 0), (37, 5, 2), (64, 8, 8), (2200, 3, 0), (512, 1, 8)):
        mu = 0.5 + torch.randn(n_mix, W, generator=g)
        state = torch.zeros(4, W + 5, device="cuda")
        last = {s: np.zeros(W) for s in range(4)}
        for plan in ([(2, 1), (0, 9), (3, 2)], [(0, 1), (1, 1), (2, 1)], [(3, 30), (2, 3)], [(1, 2), (0, 17), (3, 1)]):
            T = sum(n for _, n in plan)
            h = rounded(torch.randn(T + 2, W + pad, generator=g), dtype)
            seq = torch.tensor([i for i, (_, n) in enumerate(plan) for _ in range(n)] + [-1, -1], dtype=torch.int32, device="cuda")
            cu = torch.tensor(np.cumsum([0] + [n for _, n in plan]), dtype=torch.int32, device="cuda")
            out = torch.full((T + 2, n_mix * W), 3.0, dtype=DTYPES[dtype], device="cuda")
            ops.token_shift(dev(h.float(), dtype)[:, :W], state, ints(*[s for s, _ in plan]), seq, cu, mu.cuda(), out)
            got, at = out.double().cpu().numpy(), 0
            for s, n in plan:
                x = h[at:at + n, :W].numpy()
                before = pv.shifted(x, last[s])
                for m in range(n_mix):
                    ref = pv.blend(x, before, mu[m].numpy())
                    assert np.abs(got[at:at + n, m * W:(m + 1) * W] - ref).max() < (2e-6 if dtype == "float32" else 1e-2) * np.abs(ref).max(), (W, s, m)
                last[s] = x[-1]
                at += n
            assert np.abs(got[T:]).max() == 0
            for s in range(4):
                assert np.array_equal(state[s, :W].double().cpu().numpy(), last[s]) and float(state[s, W:].abs().max()) == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_products_of_blends_side_by_side(dtype):
    """One weight-streaming product for a few rows (groups whose width is a multiple of 16), batched products else; the last,
    narrower group goes through tanh and the others do not."""
    from cbis_b200.kernels import ops
    g = torch.Generator().manual_seed(3)
    for T, K, N, R in ((1, 64, 32, 8), (7, 256, 48, 48), (16, 2048, 64, 13), (5, 64, 40, 8), (40, 64, 32, 16), (9, 36, 20, 5), (3, 512, 2048, 64), (12, 64, 16, 30)):
        x = rounded(torch.randn(T, 5 * K, generator=g), dtype)
        w = rounded(torch.randn(4 * N + R, K, generator=g) * K ** -0.5, dtype)
        a, b = ops.linear_blends(dev(x.float(), dtype), dev(w.float(), dtype), 4, N, "tanh")
        ref = torch.cat([x[:, i * K:(i + 1) * K] @ w[i * N:(i + 1) * N].T for i in range(4)], 1)
        tail = torch.tanh(x[:, 4 * K:] @ w[4 * N:].T)
        tol = 1e-5 if dtype == "float32" else 2e-2
        assert a.shape == (T, 4 * N) and b.shape == (T, R)
        assert (a.double().cpu() - ref).abs().max() < tol * ref.abs().max() and (b.double().cpu() - tail).abs().max() < tol, (T, K, N, R)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H, D", [(3, 8), (2, 16), (1, 5), (4, 20), (2, 33), (2, 64), (1, 96), (1, 128), (1, 200), (1, 300)])
def test_the_recurrence_over_steps(H, D, dtype):
    """Segments of unlike lengths (one row, two, batches' edges, long) over several steps, slots used again; decays from
    near zero to so near one that a rounded decay would lose them; whole, and cut into pieces that run side by side."""
    from cbis_b200.kernels import ops
    g = torch.Generator().manual_seed(4)
    HD, stride = H * D, -(-H * D * D // 4) * 4 + 8
    w0 = 4.0 * torch.randn(HD, generator=g) - 3.0
    w0[::5] = -14.0                                   # hardly any decay
    u = torch.randn(H, D, generator=g)
    for piece in (0, 16, 48):
        state = torch.zeros(4, stride, device="cuda")
        kept = {s: None for s in range(4)}
        for plan in ([(2, 1), (0, 70), (3, 2)], [(0, 1), (1, 4), (2, 1)], [(3, 33), (2, 16), (1, 17)], [(0, 129)]):
            T = sum(n for _, n in plan)
            x = rounded(torch.randn(T, 3 * HD + 7, generator=g), dtype)
            raw = torch.randn(T, HD + 3, generator=g)
            cu = torch.tensor(np.cumsum([0] + [n for _, n in plan]), dtype=torch.int32, device="cuda")
            y = torch.zeros(T, HD, device="cuda")
            ops.time_mixing(dev(x.float(), dtype), 1, 4 + HD, 6 + 2 * HD, raw.cuda()[:, :HD], w0.cuda(), u.reshape(-1).cuda(), state,
                            ints(*[s for s, _ in plan]), cu, len(plan), H, D, y, max_seg_rows=max(n for _, n in plan), piece_rows=piece)
            got, at = y.double().cpu().numpy(), 0
            w = np.exp(-np.exp(raw[:, :HD].double().numpy() + w0.double().numpy())).reshape(T, H, D)
            for s, n in plan:
                r, k, v = (x[at:at + n, c:c + HD].numpy().reshape(n, H, D) for c in (1, 4 + HD, 6 + 2 * HD))
                ref, kept[s] = pv.recurrence(r, k, v, w[at:at + n], u.numpy(), kept[s])
                err = np.abs(got[at:at + n] - ref.reshape(n, HD)).max()
                assert err < 2e-5 * max(1.0, np.abs(ref).max()), (piece, s, n, err)
                S = state[s, :HD * D].double().cpu().numpy().reshape(H, D, D).transpose(0, 2, 1)
                assert np.abs(S - kept[s]).max() < 2e-5 * max(1.0, np.abs(kept[s]).max())
                at += n
        assert float(state[:, -(-HD * D // 4) * 4:].abs().max()) == 0


def test_a_long_prompt_beside_decoding_rows_is_cut_into_pieces():
    from cbis_b200.kernels import ops
    g = torch.Generator().manual_seed(5)
    H, D, lens = 2, 32, [1, 1, 300]
    T = sum(lens)
    assert ops.time_mixing_piece_rows(300, 3, H, D, total_rows=T) > 0
    x, raw = torch.randn(T, 3 * H * D, generator=g), torch.randn(T, H * D, generator=g)
    w0, u = torch.randn(H * D, generator=g) - 4.0, torch.randn(H * D, generator=g)
    cu = torch.tensor([0, 1, 2, T], dtype=torch.int32, device="cuda")
    outs = []
    for piece in (None, 0):
        state, y = torch.ones(3, H * D * D, device="cuda"), torch.zeros(T, H * D, device="cuda")
        ops.time_mixing(x.cuda(), 0, H * D, 2 * H * D, raw.cuda(), w0.cuda(), u.cuda(), state, ints(2, 0, 1), cu, 3, H, D, y, max_seg_rows=300, piece_rows=piece)
        outs.append((y, state))
    assert (outs[0][0] - outs[1][0]).abs().max() < 1e-4 * outs[1][0].abs().max() and (outs[0][1] - outs[1][1]).abs().max() < 1e-4 * outs[1][1].abs().max()


# heads, key/value heads, key width, value width, page size
SHAPES = [(4, 2, 16, 16, 8), (6, 2, 24, 40, 8), (8, 2, 64, 64, 16), (4, 2, 128, 128, 16), (5, 5, 20, 12, 8), (10, 1, 80, 48, 16),
          (3, 1, 136, 200, 16), (12, 3, 48, 48, 4), (2, 1, 64, 64, 128), (2, 2, 96, 112, 32)]
# window, first keys kept, cap
MASKS = [(0, 0, 4.0), (40, 21, 0.0), (130, 5, 30.0), (1, 3, 2.0), (30, 100, 8.0), (65, 64, 5.0), (16, 0, 3.0), (200, 190, 40.0)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window, keep, cap", MASKS)
@pytest.mark.parametrize("H, G, D, V, ps", SHAPES)
def test_keys_that_stand_out_under_a_cap_and_a_window_that_keeps_first_keys(H, G, D, V, ps, window, keep, cap, dtype):
    """One sequence of 330 keys in scattered pages.  Every 29th key stands out for every query, the last kept key and the
    first one not kept too: a row hangs on the ones it sees, so a window or kept run that is one key off shows.  Pages no
    later query may read are not there (their entries of the block table are negative).  Scores reach six: caps below it
    bend them by much (the exponential form of the prefill kernel's tanh), caps far above by little (its polynomial).  Every row of
    every kernel: general (whole, keys cut), tiled tensor-core (whole, keys cut), TMA + tcgen05 (whole, keys cut), decoding
    with and without splits."""
    from cbis_b200.kernels import ops
    g = torch.Generator().manual_seed(8)
    T, scale = 330, 0.5
    direction = torch.randn(D, generator=g)
    direction /= direction.norm()
    q = rounded(0.3 * torch.randn(T, H, D, generator=g) + 3.5 * direction, dtype)
    k = 0.3 * torch.randn(T, G, D, generator=g)
    k[::29] += 3.5 * direction
    for j in (keep - 1, keep):
        if 0 <= j < T and j % 29:
            k[j] += 3.5 * direction
    k, v = rounded(k, dtype), rounded(torch.randn(T, G, V, generator=g), dtype)
    mask = {"size": window, "keep_first": keep} if window else None
    ref = torch.from_numpy(pv.attention_rows(q.numpy(), k.numpy(), v.numpy(), scale, np.arange(T), cap, mask)).view(T, H * V)
    kp, vp, bt = _paged(k, v, ps, g)

    def table(first_row):
        """The pages that the queries from ``first_row`` on may need; the others' entries are negative."""
        b = bt.clone()
        for lp in range(b.shape[1]):
            if window and lp * ps >= keep and (lp + 1) * ps <= first_row - window + 1:
                b[0, lp] = -1
        return b
    kd, vd, qd = dev(kp, dtype), dev(vp, dtype), dev(q.view(T, H * D).float(), dtype)
    pos = torch.arange(T, dtype=torch.int32, device="cuda")
    seq = torch.zeros(T, dtype=torch.int32, device="cuda")
    tol = (2e-5 if dtype == "float32" else 2.5e-2) * max(1.0, ref.abs().max().item())
    kw = dict(cap=cap, keep=keep)

    def fresh(n=T):
        return torch.zeros(n, H * V, dtype=DTYPES[dtype], device="cuda")

    def check(out, rows=slice(None), what=""):
        err = (out.double().cpu() - ref[rows]).abs().max(1).values
        assert err.max() < tol, (what, int(err.argmax()), err.max().item())

    out = fresh()
    ops.paged_attention_generic(qd, kd, vd, table(0), seq, pos, out, H, G, D, ps, scale, window, v_head_dim=V, **kw)
    check(out, what="general")
    part = torch.full((120 * H * 6 * (max(D, V) + 4),), float("nan"), device="cuda")
    if V % 4 == 0:
        for chunk in (128, 64):
            some = fresh(120)
            ops.paged_attention_generic(qd[210:], kd, vd, table(210), seq[210:], pos[210:], some, H, G, D, ps, scale, window, (-(-T // chunk), chunk), part, v_head_dim=V, **kw)
            check(some, slice(210, T), "general, keys cut")
    if dtype != "bfloat16" or D % 8 or V % 8:
        return
    cu, start = ints(0, T), ints(0)
    cu2, start2 = ints(210, T), ints(210)
    kernels = [("tiled", ops.paged_prefill_bf16, dict(v_head_dim=V, **kw))] if max(D, V) <= 128 else []
    if D == V and D in (64, 128):
        kernels.append(("TMA + tcgen05", ops.paged_prefill_tc5, kw))
    for name, fn, opts in kernels:
        out = fresh()
        fn(qd, kd, vd, table(0), cu, start, out, 0, 1, T, H, G, D, ps, scale, window, **opts)
        check(out, what=name)
        out = fresh()
        fn(qd, kd, vd, table(210), cu2, start2, out, 0, 1, 120, H, G, D, ps, scale, window, **opts)
        check(out[210:], slice(210, T), name + ", a later portion")
        for chunk in (128, 64):
            out = fresh()
            fn(qd, kd, vd, table(210), cu2, start2, out, 0, 1, 120, H, G, D, ps, scale, window, (-(-T // chunk), chunk), part, pos, 210, 120, **opts)
            check(out[210:], slice(210, T), name + ", keys cut")
    ops.raise_if_kernel_errors()
    rows = list(range(0, T, 7)) + list(range(280, 310))             # decoding rows at many positions, as one batch
    n, idx = len(rows), torch.tensor(rows, device="cuda")
    qr, pr = qd[idx].contiguous(), pos[idx].contiguous()
    tables = torch.cat([table(r) for r in rows]).contiguous()
    rs = torch.arange(n, dtype=torch.int32, device="cuda")
    for nsplit in (1, 3, 8):
        counters = torch.zeros(n * H, dtype=torch.int32, device="cuda")
        out = fresh(n)
        scratch = torch.empty(max(1, ops.decode_scratch_floats(n, H, V, nsplit)), device="cuda")
        ops.paged_decode_bf16(qr, -1, -1, kd, vd, tables, rs, pr, pr, out, scratch, counters, H, G, D, ps, scale, window, nsplit, v_head_dim=V, **kw)
        check(out, rows, f"decoding, {nsplit} splits")
        assert int(counters.abs().sum()) == 0


def test_kept_keys_behind_blocks_of_positions():
    """The mask's other kind: with blocks of 32 positions a query sees its own block and the first 10 keys (32-bit)."""
    from cbis_b200.kernels import ops
    g = torch.Generator().manual_seed(9)
    T, H, G, D, ps = 100, 2, 1, 16, 8
    q, k, v = torch.randn(T, H, D, generator=g), torch.randn(T, G, D, generator=g), torch.randn(T, G, D, generator=g)
    kp, vp, bt = _paged(k, v, ps, g)
    out = torch.zeros(T, H * D, device="cuda")
    pos = torch.arange(T, dtype=torch.int32, device="cuda")
    ops.paged_attention_generic(q.view(T, -1).cuda(), kp.cuda(), vp.cuda(), bt, torch.zeros_like(pos), pos, out, H, G, D, ps, 0.3, -32, keep=10)
    ref = []
    for i in range(T):
        see = [j for j in range(i + 1) if j >= i - i % 32 or j < 10]
        w = torch.softmax(torch.einsum("hd,jd->hj", q[i].double(), k[see, 0].double()) * 0.3, -1)
        ref.append((w @ v[see, 0].double()).reshape(-1))
    assert (out.double().cpu() - torch.stack(ref)).abs().max() < 1e-5


def test_what_the_kernels_refuse():
    """A group width the product cannot cut at, heads beyond a kernel's limits, too many blends, a cap together with a bias
    that grows with the logarithm: a message, no launch."""
    from cbis_b200.kernels import ops
    z = lambda *s, t=torch.bfloat16: torch.zeros(*s, dtype=t, device="cuda")
    f = lambda *s: z(*s, t=torch.float32)
    i = lambda *s: torch.zeros(*s, dtype=torch.int32, device="cuda")
    with pytest.raises(ops.KernelError, match="size"):
        ops.gemm_small_m(z(4, 2 * 64), z(48, 64), None, None, z(4, 48), group_n=24)
    with pytest.raises(ops.KernelError, match="size"):
        ops.qk_turn_norm(z(2, 600), 0, 1, 600, 0, 600, 1e-5, i(2), None, 0)
    with pytest.raises(ops.KernelError, match="size"):
        ops.token_shift(z(2, 8), f(1, 8), i(1), i(2), i(2), f(9, 8), z(2, 72))
    with pytest.raises(ops.KernelError, match="size"):
        ops.time_mixing(f(2, 3 * 600), 0, 600, 1200, f(2, 600), f(600), f(600), f(1, 600 * 600), i(1), i(2), 1, 1, 600, f(2, 600))
    k = z(4, 2, 16, 64)
    with pytest.raises(ops.KernelError, match="size"):
        ops.paged_prefill_tc5(z(32, 4 * 64), k, k.clone(), i(1, 4), i(2), i(1), z(32, 4 * 64), 0, 1, 32, 4, 2, 64, 16, 1.0, cap=3.0, slopes=f(4), rates=f(4))
