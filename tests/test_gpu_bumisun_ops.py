"""The kernels behind the Bumisun parts, each against the plain implementation's functions or a few lines of float64."""
import numpy as np
import pytest
import torch

import plain_bumisun as plain
from test_gpu_dobelix_ops import DEV, make_step
from test_gpu_pupinex_ops import _paged, close, dev, token_step

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


def wide(t):
    return t.float().cpu().numpy().astype(np.float64)


# ------------------------------------------------------------------ embedding, gates, router
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [6, 64, 1500, 5000])
def test_embedding_and_its_norm(dtype, width):
    from hfee_b200.kernels import ops
    rng = np.random.default_rng(width)
    table, w = dev(rng.normal(size=(30, width)), dtype), dev(rng.normal(size=width) + 1.0)
    step = token_step([(1, [3, 29, 0, -1]), (3, [7])], [0, 0, 0, 0])
    feedback = dev([4, 12, 9, 2], torch.int32)                     # token -1: what the device sampled last for the slot
    out = torch.empty((5, width), device=DEV)
    ops.embed_norm(table, step.token_ids, w, 1e-3, out, step.slot_of_token, feedback)
    assert close(wide(out), plain.rms_norm(wide(table)[[3, 29, 0, 12, 7]], wide(w), 1e-3), 3e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,parts", [(64, 1), (96, 4), (21, 3), (5000, 1), (9216, 2), (40, 40), (1200, 8)])
def test_gate_in_front_of_a_norm_in_parts(dtype, width, parts):
    """Parts of very different size, so that a shared root mean square would show."""
    from hfee_b200.kernels import ops
    rng = np.random.default_rng(width + parts)
    n, eps = 7, 1e-2
    x = rng.normal(size=(n, width)) * np.repeat(10.0 ** rng.uniform(-1.5, 1.5, size=parts), width // parts)
    z = dev(rng.normal(size=(n, width + 5)) * 2, dtype)[:, 3:width + 3]
    w = rng.normal(size=width) + 1.0
    buf = torch.zeros((n, width + 4), dtype=dtype, device=DEV)
    ops.gate_parts_norm(dev(x), z, dev(w), eps, parts, buf[:, :width], 0.5)
    want = 0.5 * plain.norm_in_parts(x * plain.silu(wide(z)), w, eps, parts)
    assert close(wide(buf[:, :width]), want, 4e-6 if dtype == torch.float32 else 8e-3) and torch.count_nonzero(buf[:, width:]) == 0


@pytest.mark.parametrize("experts,top", [(4, 1), (16, 3), (7, 7), (64, 40), (130, 2)])
def test_router_weights_over_the_chosen_logits(experts, top):
    from hfee_b200.kernels import ops
    rng = np.random.default_rng(experts)
    n = 11
    z = np.round(rng.normal(size=(n, experts)) * 4, 1)             # ties happen: the lower expert goes first
    z[3] *= 40.0                                                   # logits far apart: weights underflow to zero
    b = np.round(rng.normal(size=experts), 1)
    logits = torch.full((n, experts + 2), 1e9, device=DEV)         # columns behind the experts are not the router's
    logits[:, :experts] = dev(z)
    choice, weight = torch.empty((n, top), dtype=torch.int32, device=DEV), torch.empty((n, top), device=DEV)
    for bias in (None, b):
        ops.moe_route_chosen(logits, experts, top, 1.5, choice, weight, None if bias is None else dev(bias))
        total = (z.astype(np.float32) + (0 if bias is None else bias.astype(np.float32))).astype(np.float64)
        want, share = plain.choose(total, top)
        assert np.array_equal(choice.cpu().numpy(), want) and close(wide(weight), 1.5 * share, 1e-6)


@pytest.mark.parametrize("m", [1, 2, 5, 8, 12, 40, 64, 70, 300])
@pytest.mark.parametrize("inner,k", [(96, 64), (640, 512)])
def test_relu_gate_in_the_epilogues(m, inner, k):
    """relu(gate) * up for every number of rows that takes another product kernel, and in float32."""
    from hfee_b200.kernels import ops
    rng = np.random.default_rng(m)
    a, gate, up = rng.normal(size=(m, k)), rng.normal(size=(inner, k)) * k ** -0.5, rng.normal(size=(inner, k)) * k ** -0.5
    for dtype, tol in ((torch.bfloat16, 1e-2), (torch.float32, 1e-5)):
        ad, gd, ud = dev(a, dtype), dev(gate, dtype), dev(up, dtype)
        want = np.maximum(wide(ad) @ wide(gd).T, 0.0) * (wide(ad) @ wide(ud).T)
        granule = ops.SWIGLU_GRANULE if dtype == torch.bfloat16 else inner
        w = ops.interleave_gate_up(gd, ud, granule)
        out, scratch = torch.empty((m, inner), dtype=dtype, device=DEV), torch.empty((m, 2 * inner), dtype=dtype, device=DEV)
        ops.linear_gated_normed(ad, w, out, granule, scratch, "relu")
        assert close(wide(out), want, tol), dtype
        ops.linear(ad, w, scratch)
        ops.gated_act(scratch, out, "relu", granule)
        assert close(wide(out), want, 2 * tol), dtype


def test_relu_gate_on_paired_tiles():
    from hfee_b200.kernels import ops
    torch.manual_seed(0)
    a, w = torch.randn(520, 128, device=DEV).bfloat16(), (torch.randn(8192, 128, device=DEV) * 0.1).bfloat16()
    ref = (a.float() @ w.float().t()).reshape(520, 1024, 2, 4)
    want = (ref[:, :, 0].clamp(min=0) * ref[:, :, 1]).reshape(520, 4096)
    for run in (ops.gemm_tcgen05_pair, lambda *x: ops.gemm_tcgen05(*x, block_n=128)):
        out = torch.empty((520, 4096), dtype=torch.bfloat16, device=DEV)
        run(a, w, out, ops.EPI_REGLU)
        assert close(wide(out), wide(want), 1e-2)
    ops.check_status()


# ------------------------------------------------------------------ attention
def plain_attention(q, k, v, scale, size, keep, softcap, sink):
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        s = plain.cap((q[:, h] @ k[:, h // (H // G)].T) * scale, softcap)
        w = plain.sink_softmax(np.where(plain.visible(T, size, keep), s, -np.inf), sink[h])
        out[:, h] = w @ v[:, h // (H // G)]
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("page", [16, 64])
@pytest.mark.parametrize("heads,kv,dim,vdim,window,keep,softcap", [
    (4, 2, 16, 24, 21, 5, 2.0), (2, 2, 64, 64, 200, 7, None), (6, 1, 32, 8, 1, 1, 5.0), (3, 3, 12, 10, 40, 33, 1.5), (8, 2, 128, 64, 77, 70, 30.0),
    (4, 4, 32, 96, 64, 64, 8.0), (2, 1, 16, 16, 90, 0, 3.0), (4, 1, 48, 16, None, 0, 1.0), (16, 2, 64, 64, 30, 200, 4.0), (8, 1, 128, 128, 65, 3, 6.0)])
def test_windows_that_keep_the_first_tokens(dtype, page, heads, kv, dim, vdim, window, keep, softcap):
    """Prompt portions behind cached tokens, single decoded tokens (keys split among thread blocks where the kernel does
    that) and short ones, with every page that neither the window nor the kept tokens need taken out of the block table."""
    from hfee_b200.kernels import ops
    rng = np.random.default_rng(heads + dim + keep)
    T = 430
    q, k, v = rng.normal(size=(T, heads, dim)), rng.normal(size=(T, kv, dim)), rng.normal(size=(T, kv, vdim))
    sink = rng.uniform(-2.0, 3.0, size=heads)
    scale = 1.5 * dim ** -0.5
    rd = lambda a: wide(dev(a, dtype))
    want = plain_attention(rd(q), rd(k), rd(v), scale, window, keep, softcap, sink)
    pages = -(-T // page)
    order = rng.permutation(pages).tolist()
    k_pool, v_pool = _paged(k, v, page, dtype, order)
    tile = ops.distance_attention_tile(dim, vdim)
    scratch = torch.empty((4 * heads * ops.MAX_SPLITS * (tile + 2),), device=DEV) if tile else None
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    for lo, hi, splits in ((0, T, None), (0, 37, None), (37, 400, None), (429, 430, 5), (429, 430, 1), (300, 301, None), (64, 65, 3), (127, 130, None),
                           (200, 265, None)):
        table = torch.full((4, pages + 2), -1, dtype=torch.int32, device=DEV)
        row = list(order)
        if window is not None:
            for p in range(-(-keep // page), max(0, lo + 1 - window) // page):
                row[p] = pages                                         # a page of stale content that nothing may read
        table[2, :pages] = dev(row, torch.int32)
        step = make_step([hi - lo], lengths=[lo], slots=[2])
        step.attention_splits = splits
        out = torch.empty((hi - lo, heads * vdim), dtype=dtype, device=DEV)
        ops.softmax_attention(dev(q[lo:hi].reshape(hi - lo, heads * dim), dtype), k_pool, v_pool, table, page, step, out, heads, kv, dim,
                              vdim, scale, window or 0, dev(sink), 1.0, scratch, keep, softcap)
        assert close(wide(out), want[lo:hi].reshape(hi - lo, -1), tol), (lo, hi)
    ops.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
def test_edges_of_window_and_kept_tokens_to_the_key(dtype):
    """One key stands out by itself: its weight shows whether it is seen, at the window's edge and at the last kept token."""
    from hfee_b200.kernels import ops
    page, T, dim, window, keep = 16, 200, 16, 50, 11
    k, v = np.zeros((T, 1, dim)), np.zeros((T, 1, dim))
    q = np.zeros((T, 1, dim)); q[:, 0, 0] = 1.0
    for special in (0, 10, 11, 12, 63, 64, 100, 149, 150, 151):
        k[:], v[:] = 0.0, 0.0
        k[special, 0, 0], v[special, 0, 1] = 12.0, 1.0
        k_pool, v_pool = _paged(k, v, page, dtype, list(range(13)))
        table = torch.full((2, 14), -1, dtype=torch.int32, device=DEV)
        table[1, :13] = torch.arange(13, dtype=torch.int32, device=DEV)
        for lo, hi in ((0, T), (199, 200), (special + window - 1, min(T, special + window + 1)), (150, 200)):
            if lo >= T or hi > T:
                continue
            step = make_step([hi - lo], lengths=[lo], slots=[1])
            out = torch.empty((hi - lo, dim), dtype=dtype, device=DEV)
            ops.softmax_attention(dev(q[lo:hi, 0], dtype), k_pool, v_pool, table, page, step, out, 1, 1, dim, dim, 1.0, window, None, 1.0, None,
                                  keep, 100.0)
            i = np.arange(lo, hi)
            seen = (i >= special) & ((i - special < window) | (special < keep))
            got = wide(out)[:, 1]
            assert np.all(got[seen] > 0.9) and np.all(got[~seen] == 0.0), (special, lo)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim", [(4, 2, 16, 24), (3, 3, 10, 6)])
def test_values_are_mixed_before_they_are_cached(dtype, heads, kv, dim, vdim):
    from hfee_b200.kernels import ops
    rng = np.random.default_rng(dim)
    page, n, qc, kc, vc = 16, 21, heads * dim, kv * dim, kv * vdim
    table = torch.tensor([[1, 0]], dtype=torch.int32, device=DEV)
    step = make_step([n], lengths=[0], slots=[0])
    first = torch.full((n, vc), 7.0, dtype=dtype, device=DEV)
    cached = []
    src = [dev(rng.normal(size=(n, qc + kc + vc)), dtype) for _ in range(3)]
    for x, mode, share in zip(src, (ops.VALUES_STORE_FIRST, ops.VALUES_MIX, ops.VALUES_MIX), (0.9, 0.25, 1.5)):
        kp, vp = torch.zeros((2, kv, page, dim), dtype=dtype, device=DEV), torch.zeros((2, kv, page, vdim), dtype=dtype, device=DEV)
        ops.attention_prepare(x, 0, qc, qc + kc, heads, kv, dim, vdim, step, torch.empty((n, qc), dtype=dtype, device=DEV), kp, vp, table, page,
                              first_values=first, value_mix=mode, share=share)
        cached.append(wide(vp)[[1, 0]].transpose(0, 2, 1, 3).reshape(2 * page, vc)[:n])
    v = [wide(x)[:, qc + kc:] for x in src]
    assert np.array_equal(cached[0], v[0]) and np.array_equal(wide(first), v[0])
    tol = 1e-6 if dtype == torch.float32 else 5e-3
    assert close(cached[1], plain.mix_values(v[1], v[0], 0.25), tol) and close(cached[2], plain.mix_values(v[2], v[0], 1.5), tol)


# ------------------------------------------------------------------ the scan
def plain_scan(x, B, C, z, bias, a_log, d, S):
    """One request, token by token, from the state S [H, N, dv] (changed in place)."""
    T, H, dv = x.shape
    share = np.arange(H) // (H // B.shape[1])
    out = np.zeros_like(x)
    dt = plain.softplus(z + bias)
    for t in range(T):
        S *= np.exp(-np.exp(a_log) * dt[t])[:, None, None]
        S += dt[t][:, None, None] * B[t][share][:, :, None] * x[t][:, None, :]
        out[t] = np.einsum("hnc,hn->hc", S, C[t][share]) + d[:, None] * x[t]
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,groups,state,vdim", [(4, 1, 32, 48), (2, 2, 16, 8), (6, 3, 24, 40), (8, 2, 128, 64), (3, 1, 5, 33), (2, 1, 256, 96),
                                                     (1, 1, 8, 136), (4, 2, 72, 16)])
@pytest.mark.parametrize("decays", ["slow", "mixed", "strong"])
def test_head_scan_continues_across_portions(dtype, heads, groups, state, vdim, decays):
    """Portions of one and two tokens, of a run, of runs and a part, several requests in slots out of order, whichever kernels
    a step takes; strong decays underflow and must not be divided by."""
    from hfee_b200.kernels import ops
    rng = np.random.default_rng(heads * state + vdim)
    inner, bc = heads * vdim, groups * state
    lo, hi = {"slow": (-8.0, -5.0), "mixed": (-4.0, 1.5), "strong": (3.0, 5.0)}[decays]
    a_log, bias, d = rng.uniform(lo, hi, size=heads), rng.uniform(-3.0, 1.0, size=heads), rng.normal(size=heads)
    ld = -(-(inner + 2 * bc) // 8) * 8
    total = {0: 300, 2: 131, 3: 70}
    data = {s: (rng.normal(size=(T, inner + 2 * bc)) * 0.7, rng.normal(size=(T, heads))) for s, T in total.items()}
    S = torch.full((4, heads, state, vdim), 0.0, device=DEV)
    S[1] = 5.0                                                        # another request's state
    ref_S = {s: np.zeros((heads, state, vdim)) for s in total}
    at = {s: 0 for s in total}
    ws = torch.empty((ops.head_scan_workspace(4, 512, heads, state, vdim),), device=DEV)
    tol = 1e-4 if dtype == torch.float32 else 2e-4                    # bfloat16: the inputs are rounded for both
    for sizes in ({0: 130, 3: 1}, {2: 2}, {0: 1, 2: 64, 3: 65}, {0: 25, 2: 65}, {0: 144, 3: 4}):
        xs, zs = [], []
        for s, n in sizes.items():
            xs.append(data[s][0][at[s]:at[s] + n]); zs.append(data[s][1][at[s]:at[s] + n])
        n = sum(sizes.values())
        buf = torch.zeros((n, ld), dtype=dtype, device=DEV)
        buf[:, :inner + 2 * bc] = dev(np.concatenate(xs), dtype)
        zd = dev(np.concatenate(zs), dtype)
        step = make_step(list(sizes.values()), lengths=[at[s] for s in sizes], slots=list(sizes))
        out = torch.empty((n, inner), device=DEV)
        x, B, C = buf[:, :inner], buf[:, inner:inner + bc], buf[:, inner + bc:inner + 2 * bc]
        ops.head_scan(x, B, C, zd, dev(bias), dev(a_log), dev(d), S, step, out, heads, groups, state, vdim, True, ws)
        row = 0
        for s, k in sizes.items():
            r = slice(row, row + k)
            want = plain_scan(wide(x)[r].reshape(k, heads, vdim), wide(B)[r].reshape(k, groups, state), wide(C)[r].reshape(k, groups, state),
                              wide(zd)[r], bias, a_log, d, ref_S[s])
            assert close(wide(out)[r], want.reshape(k, inner), tol), (sizes, s)
            assert close(wide(S[s]), ref_S[s], tol), (sizes, s)
            at[s] += k; row += k
    assert torch.all(S[1] == 5.0)


def test_head_scan_without_a_write_leaves_the_state():
    from hfee_b200.kernels import ops
    torch.manual_seed(1)
    for n in (1, 40, 100):
        buf, z = torch.randn(n, 2 * 16 + 2 * 8, device=DEV).bfloat16(), torch.randn(n, 2, device=DEV).bfloat16()
        one, S = torch.ones(2, device=DEV), torch.randn(2, 2, 8, 16, device=DEV)
        before = S.clone()
        ws = torch.empty((ops.head_scan_workspace(2, 128, 2, 8, 16),), device=DEV)
        out = torch.empty((n, 32), device=DEV)
        ops.head_scan(buf[:, :32], buf[:, 32:40], buf[:, 40:], z, one, -one, one, S, make_step([n], lengths=[3], slots=[1]), out, 2, 1, 8, 16,
                      False, ws)
        assert torch.equal(S, before)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("interleaved", [False, True])
@pytest.mark.parametrize("heads,kv,dim,vdim,rope", [(4, 2, 32, 24, 16), (6, 2, 64, 16, 64), (2, 1, 16, 8, 8), (3, 3, 8, 40, 0), (2, 2, 128, 64, 32), (5, 1, 24, 16, 6)])
def test_attention_prepare_in_whole_pieces(dtype, interleaved, heads, kv, dim, vdim, rope):
    """Without biases and norms the preparation moves 16-byte pieces where it can; few tokens and many, over pages in any order."""
    from hfee_b200.kernels import ops
    rng = np.random.default_rng(heads * dim + rope)
    qc, kc, vc = heads * dim, kv * dim, kv * vdim
    for n, n0, page in ((1, 37, 16), (13, 21, 16), (600, 5, 64)):
        src = dev(rng.normal(size=(n, qc + kc + vc)), dtype)
        x = wide(src)
        pages = -(-(n0 + n) // page)
        order = rng.permutation(pages)
        table = torch.full((3, pages + 1), -1, dtype=torch.int32, device=DEV)
        table[1, :pages] = dev(order, torch.int32)
        step = make_step([n], lengths=[n0], slots=[1])
        cs = None
        if rope:
            inv = torch.tensor([300.0 ** (-2.0 * i / rope) for i in range(rope // 2)], dtype=torch.float64, device=DEV)
            cs = torch.empty((n, rope // 2, 2), device=DEV)
            ops.rope_table(step.positions, inv, cs)
        kp, vp = (torch.zeros((pages, kv, page, d), dtype=dtype, device=DEV) for d in (dim, vdim))
        q_out = torch.empty((n, qc), dtype=dtype, device=DEV)
        ops.attention_prepare(src, 0, qc, qc + kc, heads, kv, dim, vdim, step, q_out, kp, vp, table, page, cs, rope, interleaved)

        def rotated(t, h):
            t = t.reshape(n, h, dim).copy()
            a = (np.arange(n0, n0 + n)[:, None] * 300.0 ** (-2.0 * np.arange(rope // 2) / max(rope, 1)))[:, None, :]
            first, second = ((slice(0, rope, 2), slice(1, rope, 2)) if interleaved else (slice(0, rope // 2), slice(rope // 2, rope)))
            u, v = t[..., first].copy(), t[..., second].copy()
            t[..., first], t[..., second] = u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)
            return t
        tol = 1e-6 if dtype == torch.float32 else 5e-3
        assert close(wide(q_out), rotated(x[:, :qc], heads).reshape(n, qc), tol)
        at = np.arange(n0, n0 + n)
        pg = order[at // page]
        assert close(wide(kp)[pg, :, at % page], rotated(x[:, qc:qc + kc], kv), tol)
        assert np.array_equal(wide(vp)[pg, :, at % page].reshape(n, vc), x[:, qc + kc:])
        assert torch.count_nonzero(kp[int(order[0])][:, :n0 % page if n0 < page else 0]) == 0
