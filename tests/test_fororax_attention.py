"""Both attentions of Fororax through every attention kernel, over keys made to stand out, against the plain
implementation (GPU)."""
import numpy as np
import pytest
import torch

import plain_fororax as pf
from test_fororax_kernels import DTYPES, dev, rounded

pytestmark = pytest.mark.gpu


def _paged(k, v, ps, g):
    """Keys and values of one sequence scattered over pages in a random order; returns the pages and the block table."""
    T, G, D = k.shape
    pages = -(-T // ps)
    perm = torch.randperm(pages, generator=g)
    kp, vp = torch.full((pages, G, ps, D), 7.0), torch.full((pages, G, ps, v.shape[2]), 7.0)      # token slots past the end: not zero
    for p in range(T):
        kp[perm[p // ps], :, p % ps] = k[p].float()
        vp[perm[p // ps], :, p % ps] = v[p].float()
    return kp, vp, perm.int().view(1, pages).cuda()


# heads, key/value heads, key width, value width, page size
SHAPES = [(4, 2, 16, 16, 8), (6, 2, 24, 40, 8), (8, 2, 64, 64, 16), (4, 2, 128, 128, 16), (5, 5, 20, 12, 8), (10, 1, 80, 48, 16),
          (18, 1, 32, 104, 16), (3, 1, 136, 200, 16), (12, 3, 48, 48, 4)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["log_bias", "mixed"])
@pytest.mark.parametrize("H, G, D, V, ps", SHAPES)
def test_keys_that_stand_out_through_every_kernel(H, G, D, V, ps, kind, dtype):
    """One sequence of 330 keys in scattered pages.  Every 29th key stands out for every query (the first one too), so a
    query's result hangs on those keys: near, at pages' borders, its own, and hundreds of tokens back.  With the
    logarithmic bias the scores of the standing-out keys differ by a few units between near and far, so the bias decides
    between them.  Every row of every kernel: general (whole, keys cut), tiled tensor-core (whole, keys cut), TMA + tcgen05,
    decoding with and without splits, decoding with mixed heads."""
    from cbis_b200.kernels import ops
    g = torch.Generator().manual_seed(8)
    T, scale = 330, 0.5
    direction = torch.randn(D, generator=g)
    direction /= direction.norm()
    q = rounded(0.3 * torch.randn(T, H, D, generator=g) + 3.5 * direction, dtype)
    k = 0.3 * torch.randn(T, G, D, generator=g)
    k[::29] += 3.5 * direction
    k, v = rounded(k, dtype), rounded(torch.randn(T, G, V, generator=g), dtype)
    r1, r2 = 0.2 + torch.rand(H, generator=g), 0.02 + 0.5 * torch.rand(H, generator=g)
    sinks, talk = 6.0 * torch.rand(H, generator=g), 0.4 * torch.randn(H, H, generator=g) + 0.6 * torch.eye(H)
    mixed = kind == "mixed"
    args = dict(sinks=sinks.numpy(), talk=talk.numpy()) if mixed else dict(r1=r1.numpy(), r2=r2.numpy())
    ref = torch.from_numpy(pf.attention_rows(q.numpy(), k.numpy(), v.numpy(), scale, np.arange(T), **args)).view(T, H * V)
    vh = G if mixed else 1
    kw = dict(sinks=sinks.repeat_interleave(vh).cuda(), v_heads=vh) if mixed else dict(slopes=r1.cuda(), rates=r2.cuda())
    kp, vp, bt = _paged(k, v, ps, g)
    kd, vd, qd, td = dev(kp, dtype), dev(vp, dtype), dev(q.view(T, H * D).float(), dtype), talk.cuda()
    pos = torch.arange(T, dtype=torch.int32, device="cuda")
    seq = torch.zeros(T, dtype=torch.int32, device="cuda")
    tol = (2e-5 if dtype == "float32" else 2.5e-2) * max(1.0, ref.abs().max().item())
    nh = H * vh

    def fresh(n=T):
        return torch.zeros(n, nh * V, dtype=DTYPES[dtype], device="cuda")

    def check(out, rows=slice(None), what="", is_mixed=False):
        if mixed and not is_mixed:
            r = torch.empty(out.shape[0], H * V, dtype=out.dtype, device="cuda")
            ops.mix_heads(out, td, H, G, V, r)
            out = r
        assert (out.double().cpu() - ref[rows]).abs().max() < tol, (what, (out.double().cpu() - ref[rows]).abs().max().item())

    out = fresh()
    ops.paged_attention_generic(qd, kd, vd, bt, seq, pos, out, nh, G, D, ps, scale, 0, v_head_dim=V, **kw)
    check(out, what="general")
    part = torch.empty(120 * nh * 4 * (max(D, V) + 4), device="cuda")
    if V % 4 == 0:
        some = fresh(120)
        ops.paged_attention_generic(qd[210:], kd, vd, bt, seq[210:], pos[210:], some, nh, G, D, ps, scale, 0, (3, 128), part, v_head_dim=V, **kw)
        check(some, slice(210, T), "general, keys cut")
    if dtype != "bfloat16" or D % 8 or V % 8:
        return
    cu, start = torch.tensor([0, T], dtype=torch.int32, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
    cu2, start2 = torch.tensor([210, T], dtype=torch.int32, device="cuda"), torch.full((1,), 210, dtype=torch.int32, device="cuda")
    if max(D, V) <= 128:
        out = fresh()
        ops.paged_prefill_bf16(qd, kd, vd, bt, cu, start, out, 0, 1, T, nh, G, D, ps, scale, 0, v_head_dim=V, **kw)
        check(out, what="tiled")
        out = fresh()
        ops.paged_prefill_bf16(qd, kd, vd, bt, cu2, start2, out, 0, 1, 120, nh, G, D, ps, scale, 0, (3, 128), part, pos, 210, 120, v_head_dim=V, **kw)
        check(out[210:], slice(210, T), "tiled, keys cut")
    if D == V and D in (64, 128):
        out = fresh()
        ops.paged_prefill_tc5(qd, kd, vd, bt, cu, start, out, 0, 1, T, nh, G, D, ps, scale, 0, **kw)
        check(out, what="TMA + tcgen05")
        out = fresh()
        ops.paged_prefill_tc5(qd, kd, vd, bt, cu2, start2, out, 0, 1, 120, nh, G, D, ps, scale, 0, (3, 128), part, pos, 210, 120, **kw)
        check(out[210:], slice(210, T), "TMA + tcgen05, keys cut")
        ops.raise_if_kernel_errors()
    rows = list(range(0, T, 7)) + list(range(280, 310))             # decoding rows at many positions, as one batch
    n, idx = len(rows), torch.tensor(rows, device="cuda")
    qr, pr = qd[idx].contiguous(), pos[idx].contiguous()
    for nsplit in (1, 4):
        counters = torch.zeros(n * nh, dtype=torch.int32, device="cuda")
        out = fresh(n)
        scratch = torch.empty(max(1, ops.decode_scratch_floats(n, nh, V, nsplit)), device="cuda")
        ops.paged_decode_bf16(qr, -1, -1, kd, vd, bt, seq[:n], pr, pr, out, scratch, counters, nh, G, D, ps, scale, 0, nsplit, v_head_dim=V, **kw)
        check(out, rows, f"decoding, {nsplit} splits")
        if mixed:
            cap = -(-T // 16) * 16
            scratch = torch.full((ops.decode_mix_scratch_floats(n, H, V, cap, nsplit),), float("nan"), device="cuda")
            out = torch.zeros(n, H * V, dtype=torch.bfloat16, device="cuda")
            ops.decode_mix_bf16(qr, -1, -1, kd, vd, bt, seq[:n], pr, pr, td, sinks.cuda(), None, out, scratch, counters, cap, H, G, D, V,
                                ps, scale, 0, nsplit)
            check(out, rows, f"decoding with mixed heads, {nsplit} splits", is_mixed=True)
            assert int(counters.abs().sum()) == 0


def test_decoding_with_mixed_heads_stores_keys_and_values_and_takes_the_gate():
    """The current token's key and value come from the projections and are stored; a gate; a sliding window; a padding row
    (no request) gets zeros and stores nothing."""
    from cbis_b200.kernels import ops
    g = torch.Generator().manual_seed(9)
    T, H, G, D, V, ps, scale, window = 150, 6, 2, 32, 40, 8, 0.3, 47
    bf = "bfloat16"
    k, v = rounded(torch.randn(T, G, D, generator=g), bf), rounded(torch.randn(T, G, V, generator=g), bf)
    q, gate = rounded(torch.randn(1, H, D, generator=g), bf), rounded(torch.randn(1, H * V, generator=g), bf)
    sinks, talk = torch.rand(H, generator=g), torch.randn(H, H, generator=g)
    kp, vp, bt = _paged(k, v, ps, g)
    last = int(bt[0, (T - 1) // ps])
    kp[last, :, (T - 1) % ps] = 9.0
    vp[last, :, (T - 1) % ps] = 9.0
    kd, vd = dev(kp, bf), dev(vp, bf)
    row = torch.cat([q.reshape(1, -1), k[T - 1].reshape(1, -1), v[T - 1].reshape(1, -1)], 1).float()
    qkv = dev(row.repeat(2, 1), bf)
    seq = torch.tensor([0, -1], dtype=torch.int32, device="cuda")
    pos = torch.tensor([T - 1, 0], dtype=torch.int32, device="cuda")
    slot = torch.tensor([last * ps + (T - 1) % ps, -1], dtype=torch.int32, device="cuda")
    lo = T - window
    full = np.concatenate([np.zeros((window - 1, H, D)), q.numpy()])
    ref = pf.attention_rows(full, k[lo:].numpy(), v[lo:].numpy(), scale, np.arange(window), sinks=sinks.numpy(), talk=talk.numpy())[-1]
    ref = ref.reshape(-1) * pf.sigmoid(gate.numpy()[0])
    for nsplit in (1, 3):
        out = torch.full((2, H * V), 5.0, dtype=torch.bfloat16, device="cuda")
        cap = -(-T // 16) * 16
        scratch = torch.full((ops.decode_mix_scratch_floats(2, H, V, cap, nsplit),), float("nan"), device="cuda")
        counters = torch.zeros(2 * H * G, dtype=torch.int32, device="cuda")
        before = kd.clone()
        ops.decode_mix_bf16(qkv, H * D, (H + G) * D, kd, vd, bt, seq, pos, slot, talk.cuda(), sinks.cuda(), dev(gate.repeat(2, 1).float(), bf),
                            out, scratch, counters, cap, H, G, D, V, ps, scale, window, nsplit)
        assert np.abs(out[0].double().cpu().numpy() - ref).max() < 2e-2 * np.abs(ref).max() and float(out[1].abs().max()) == 0
        assert torch.equal(kd[last, :, (T - 1) % ps].double().cpu(), k[T - 1]) and torch.equal(vd[last, :, (T - 1) % ps].double().cpu(), v[T - 1])
        before[last, :, (T - 1) % ps] = kd[last, :, (T - 1) % ps]
        assert torch.equal(before, kd)


def test_what_the_kernels_refuse():
    """Rows too narrow for the launch's heads, a matrix of another size, heads beyond a kernel's limits: a message, no
    launch."""
    from cbis_b200.kernels import ops
    z = lambda *s, t=torch.bfloat16: torch.zeros(*s, dtype=t, device="cuda")
    i = lambda *s: torch.zeros(*s, dtype=torch.int32, device="cuda")
    k = z(4, 2, 16, 64)
    for fn in (ops.paged_prefill_tc5, ops.paged_prefill_bf16):
        with pytest.raises(ops.KernelError, match="do not fit"):
            fn(z(32, 4 * 64), k, k.clone(), i(1, 4), i(2), i(1), z(32, 8 * 64), 0, 1, 32, 8, 2, 64, 16, 1.0)
    with pytest.raises(ops.KernelError, match="do not fit"):
        ops.paged_attention_generic(z(32, 4 * 64), k, k.clone(), i(1, 4), i(32), i(32), z(32, 4 * 64), 8, 2, 64, 16, 1.0, v_heads=2)
    with pytest.raises(ops.KernelError, match="size"):
        ops.qk_head_norm(z(2, 600), 0, 1, 600, 0, 600, z(600, t=torch.float32), None, 1e-5)
    with pytest.raises(AssertionError):
        ops.mix_heads(z(2, 4 * 2 * 8), z(3, 3, t=torch.float32), 4, 2, 8, z(2, 32))
