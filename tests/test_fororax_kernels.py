"""Each mechanism of Fororax through its kernels alone, against the plain implementation (GPU)."""
import numpy as np
import pytest
import torch

import plain_fororax as pf

pytestmark = pytest.mark.gpu

DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def dev(t, dtype):
    return t.to(device="cuda", dtype=DTYPES[dtype]).contiguous()


def rounded(t, dtype):
    return t.to(DTYPES[dtype]).double()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_norm_of_a_sum(dtype):
    """x = norm(alpha x + delta), the row handed on as it is or through one more norm, all rows or the wanted ones; rows
    in registers and staged in shared memory, with and without a bias on what is added."""
    from cbis_b200.kernels import ops
    g = torch.Generator().manual_seed(1)
    for width, pad in ((40, 3), (64, 4), (321, 3), (1000, 8), (2048, 0), (4100, 4)):
        x = torch.randn(9, width, generator=g) * 2
        y = rounded(torch.randn(9, width + pad, generator=g) * 5, dtype)[:, pad:]
        bias = torch.randn(width, generator=g)
        ws, wn = 1 + 0.3 * torch.randn(width, generator=g), 1 + 0.3 * torch.randn(width, generator=g)
        rows = torch.tensor([7, 0, 3], dtype=torch.int32)
        for w in (None, wn.cuda()):
            for b in (None, bias):
                x_ref = pf.norm_of_sum(x.double().numpy(), y.numpy() + (0 if b is None else b.double().numpy()), 1.7, ws.numpy(), 1e-3)
                o_ref = x_ref if w is None else pf.rms_norm(x_ref, wn.numpy(), 1e-4)
                yd = dev(torch.cat([torch.zeros(9, pad), y.float()], 1), dtype)[:, pad:]
                kw = dict(x_scale=1.7, stream=(ws.cuda(), 1e-3, 0.0))
                xd, out = x.cuda(), torch.empty(9, width, dtype=DTYPES[dtype], device="cuda")
                ops.add_rmsnorm(xd, yd, None if b is None else b.cuda(), None, w, 1e-4, 0.0, out, **kw)
                assert np.abs(xd.double().cpu().numpy() - x_ref).max() < 2e-6 * max(1.0, np.abs(x_ref).max())
                tol = (1e-5 if dtype == "float32" else 1e-2) * np.abs(o_ref).max()
                assert np.abs(out.double().cpu().numpy() - o_ref).max() < tol
                xd, some = x.cuda(), torch.empty(3, width, dtype=DTYPES[dtype], device="cuda")
                ops.add_rmsnorm(xd, yd, None if b is None else b.cuda(), None, w, 1e-4, 0.0, some, rows.cuda(), **kw)
                assert torch.equal(xd.cpu(), x) and np.abs(some.double().cpu().numpy() - o_ref[rows.numpy()]).max() < tol


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_norm_per_head(dtype):
    from cbis_b200.kernels import ops
    g = torch.Generator().manual_seed(2)
    for T, H, G, D, extra in ((5, 4, 2, 16, 8), (33, 3, 1, 20, 4), (7, 2, 2, 9, 3), (3, 5, 0, 130, 0), (2, 2, 1, 512, 4), (200, 8, 2, 128, 0)):
        n = (H + G) * D
        x = rounded(torch.randn(T, n + extra, generator=g) * 3, dtype)
        wq, wk = 1 + 0.3 * torch.randn(D, generator=g), 1 + 0.3 * torch.randn(D, generator=g)
        buf = dev(x.float(), dtype)
        ops.qk_head_norm(buf, 0, H, H * D, G, D, wq.cuda(), wk.cuda() if G else None, 1e-3)
        got = buf.double().cpu().numpy()
        heads = x[:, :n].numpy().reshape(T, H + G, D)
        ref = np.concatenate([pf.rms_norm(heads[:, :H], wq.numpy(), 1e-3), pf.rms_norm(heads[:, H:], wk.numpy(), 1e-3)], 1).reshape(T, n)
        assert np.abs(got[:, :n] - ref).max() < (1e-5 if dtype == "float32" else 3e-2), (T, H, G, D)
        assert np.array_equal(got[:, n:], x[:, n:].numpy())         # the columns behind q and k are left alone


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_results_mixed_across_heads(dtype):
    from cbis_b200.kernels import ops
    g = torch.Generator().manual_seed(3)
    for T, H, G, V in ((5, 4, 2, 16), (3, 6, 3, 7), (9, 5, 1, 12), (2, 8, 8, 24), (40, 16, 4, 128), (3, 12, 1, 9), (2, 120, 4, 8)):
        o = rounded(torch.randn(T, H, G, V, generator=g), dtype)
        t, z = torch.randn(H, H, generator=g), rounded(torch.randn(T, H * V, generator=g), dtype)
        ref = np.einsum("hg,tghv->thv", t.double().numpy(), np.stack([o[:, :, h // (H // G)].numpy() for h in range(H)], 2)).reshape(T, H * V)
        for gate in (None, z):
            out = torch.empty(T, H * V, dtype=DTYPES[dtype], device="cuda")
            ops.mix_heads(dev(o.reshape(T, -1).float(), dtype), t.cuda(), H, G, V, out, None if gate is None else dev(gate.float(), dtype))
            r = ref if gate is None else ref * pf.sigmoid(gate.numpy())
            assert np.abs(out.double().cpu().numpy() - r).max() < (1e-5 if dtype == "float32" else 6e-3) * np.abs(r).max(), (H, G, V)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_choice_is_corrected_and_the_weights_are_not(dtype):
    """Softmax scores over all outputs; a correction large enough to change the choice of most rows; the weights are the
    scores without it; the row gate is the sigmoid of one more row of the router."""
    from cbis_b200.kernels import ops
    g = torch.Generator().manual_seed(4)
    for rows, W, E, top in ((19, 40, 7, 3), (5, 64, 12, 1), (33, 24, 4, 4), (50, 72, 40, 6)):
        h = rounded(torch.randn(rows, W, generator=g), dtype)
        r = rounded(torch.randn(E + 1, W, generator=g) * 0.3, dtype)
        c = torch.randn(E, generator=g) * 0.5
        ids, weights, gap = pf.route(h.numpy(), r[:E].numpy(), c.numpy(), top)
        bare, _, _ = pf.route(h.numpy(), r[:E].numpy(), np.zeros(E), top)
        assert top == E or (np.sort(ids, 1) != np.sort(bare, 1)).any(1).mean() > 0.3
        di = torch.empty(rows, top, dtype=torch.int32, device="cuda")
        dw, side = torch.empty(rows, top, device="cuda"), torch.empty(rows, device="cuda")
        ops.route_topk(dev(h.float(), dtype), dev(r.float(), dtype), top, "softmax", False, di, dw, correction=c.cuda(), side=side)
        sure = gap > 1e-4
        assert sure.sum() > rows // 2
        og, orf = np.argsort(di.cpu().numpy(), 1), np.argsort(ids, 1)
        assert np.array_equal(np.take_along_axis(di.cpu().numpy(), og, 1)[sure], np.take_along_axis(ids, orf, 1)[sure])
        assert np.abs(np.take_along_axis(dw.cpu().numpy(), og, 1)[sure] - np.take_along_axis(weights, orf, 1)[sure]).max() < 1e-5
        assert np.abs(side.cpu().numpy() - pf.sigmoid(h.numpy() @ r[E].numpy())).max() < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_gated_products_with_cut_off_projections(dtype):
    """The limits cut both sides of the up value and only the upper side of the gate; inputs far beyond them."""
    from cbis_b200.kernels import ops
    g = torch.Generator().manual_seed(5)
    for rows, n, limit in ((21, 12, 1.0), (3, 7, 0.4), (300, 24, 2.5)):
        a, b = (rounded(torch.randn(rows, n, generator=g) * 3, dtype) for _ in range(2))
        row_gate = torch.rand(rows, generator=g)
        out = torch.empty(rows, n, dtype=DTYPES[dtype], device="cuda")
        ops.gate_mul(dev(a.float(), dtype), dev(b.float(), dtype), "silu", out, limit=limit, beta=1.702, shift=1.0, row_gate=row_gate.cuda())
        ref = pf.gated_product(a.numpy(), b.numpy(), limit) * row_gate.double().numpy()[:, None]
        assert np.abs(out.double().cpu().numpy() - ref).max() < (2e-6 if dtype == "float32" else 5e-3) * np.abs(ref).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_routed_experts_beside_identity_experts(dtype):
    """Few rows (streaming kernels) and many (tiles): a row's choices may all be experts, all identity experts or both; one
    choice a row; sums that are added to rows and sums that replace them."""
    from cbis_b200.kernels import ops
    g = torch.Generator().manual_seed(6)
    for rows, W, F, E, ident, top in ((4, 24, 16, 3, 2, 2), (70, 64, 40, 5, 3, 3), (150, 64, 24, 4, 2, 1), (40, 72, 104, 2, 1, 3), (9, 20, 12, 6, 0, 2)):
        h = rounded(torch.randn(rows, W, generator=g), dtype)
        gu, dn = rounded(torch.randn(E, 2 * F, W, generator=g) * W ** -0.5 * 2, dtype), rounded(torch.randn(E, W, F, generator=g) * F ** -0.5, dtype)
        ids = torch.stack([torch.randperm(E + ident, generator=g)[:top] for _ in range(rows)]).int()
        wt = torch.rand(rows, top, generator=g)
        ref = np.zeros((rows, W))
        for t in range(rows):
            for e, w in zip(ids[t].tolist(), wt[t].double().tolist()):
                if e >= E:
                    ref[t] += w * h[t].numpy()
                    continue
                a = pf.gated_product(gu[e, :F].numpy() @ h[t].numpy(), gu[e, F:].numpy() @ h[t].numpy(), 1.2)
                ref[t] += w * (dn[e].numpy() @ a)
        hd, gud, dnd, idd, wd = dev(h.float(), dtype), dev(gu.float(), dtype), dev(dn.float(), dtype), ids.cuda(), wt.cuda()
        kw = dict(limit=1.2, beta=1.702, shift=1.0)
        tol = (1e-5 if dtype == "float32" else 1e-2) * max(1.0, np.abs(ref).max())
        base = torch.randn(rows, W, generator=g)
        for accumulate in (False, True):
            want = ref + (base.double().numpy() if accumulate else 0)
            out, hid = base.cuda(), torch.empty(rows * top, F, dtype=DTYPES[dtype], device="cuda")
            ops.routed_gate_up(hd, gud, idd, wd, "silu", False, hid, **kw)
            ops.routed_down(hid, dnd, idd, wd, False, out, accumulate=accumulate, h=hd)
            assert np.abs(out.double().cpu().numpy() - want).max() < tol, ("streamed", rows, accumulate)
            if ops.routed_tiles_takes(hd, gud, dnd):
                out = base.cuda()
                ops.routed_tiles(hd, gud, dnd, idd, wd, "silu", False, out, accumulate=accumulate, identity=ident, **kw)
                assert np.abs(out.double().cpu().numpy() - want).max() < tol, ("tiles", rows, accumulate)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_token_rows_scaled_and_position_rows_not(dtype):
    from cbis_b200.kernels import ops
    g = torch.Generator().manual_seed(7)
    table, pos = rounded(torch.randn(30, 24, generator=g), dtype), rounded(torch.randn(50, 24, generator=g), dtype)
    toks, at = torch.randint(0, 30, (17,), generator=g).int(), torch.randint(0, 50, (17,), generator=g).int()
    out = torch.empty(17, 24, device="cuda")
    err = torch.zeros(1, dtype=torch.int32, device="cuda")
    ops.embed_pos_add(toks.cuda(), at.cuda(), dev(table.float(), dtype), dev(pos.float(), dtype), out, err, 0.35)
    ref = pf.embed({"embed": table.numpy(), "pos": pos.numpy()}, toks.tolist(), at.tolist(), 0.35)
    assert np.abs(out.double().cpu().numpy() - ref).max() < 1e-6 and int(err) == 0
