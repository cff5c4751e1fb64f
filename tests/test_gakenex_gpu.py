"""Gakenex on the GPU.  Kernels alone against their plain PyTorch statements, with inputs made so that a fault shows
(one loud key on either side of a window's edge and of the last kept position, pages that were given back in between,
two maps that answer differently, carried inputs of a convolution that are larger than the new ones, gate and up values
beyond their limits); then the engine against the plain model: single layers, configurations of unlike sizes under
every cutting in both precisions, slots and pages that are used again, long greedy decoding through the scheduler and
the replayed graphs, the command line."""
import math
from types import SimpleNamespace

import pytest
import torch

import cuttings
import plain_gakenex as plain
from gakenex_models import (CONFIGS, attention, clear_requests, dense, layer, model, moe, one_layer, ratios, references,
                            row_error, tokens, write_model)
from plain_ops import PlainOps

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def ops():
    from dlm_b200.ops import native_ops
    return native_ops(fast=True)


@pytest.fixture(scope="module")
def slow_ops():
    from dlm_b200.ops import native_ops
    return native_ops(fast=False)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("gakenex_gpu")
    out = {}
    for name, cfg in CONFIGS.items():
        folder = str(base / name)
        out[name] = (folder, plain.PlainGakenex(cfg, write_model(cfg, folder, seed=ord(name))))
    return out


def batch_of(lengths, slots, starts=None):
    """The fields of a step the kernels read, for requests that bring ``lengths`` tokens from ``starts`` on."""
    starts = starts or [0] * len(lengths)
    cu = [0]
    for n in lengths:
        cu.append(cu[-1] + n)
    i32 = dict(dtype=torch.int32, device=DEV)
    return SimpleNamespace(
        num_requests=len(lengths), num_single=sum(n == 1 for n in lengths), cu_q=torch.tensor(cu, **i32),
        state_slot=torch.tensor(slots, **i32), token_req=torch.tensor([r for r, n in enumerate(lengths) for _ in range(n)], **i32),
        positions=torch.tensor([s + i for s, n in zip(starts, lengths) for i in range(n)], **i32))


def to_cpu(b):
    return SimpleNamespace(**{k: (v.cpu() if torch.is_tensor(v) else v) for k, v in vars(b).items()})


def randn(*shape, seed=0, std=1.0, dtype=torch.float32):
    return (std * torch.randn(*shape, generator=torch.Generator().manual_seed(seed))).to(DEV, dtype)


def tol(dtype, f32=2e-5, bf16=2e-2):
    return dict(atol=f32, rtol=f32) if dtype == torch.float32 else dict(atol=bf16, rtol=bf16)


# ============================================================== attention over a window that keeps the first tokens
def paged(reqs, nkv, hd, ps, dtype, seed, window=0, keep=0):
    """reqs: [(kv_len, q_len)].  Pages scattered over the pool; a page in which no query of the step sees anything has
    been given back (-1 in the table), and what it held is still in the pool.  Returns k, v, table, cu_q, kv_len, and the
    whole table as it was."""
    total = sum(-(-n // ps) for n, _ in reqs) + 3
    perm = torch.randperm(total, generator=torch.Generator().manual_seed(seed)).tolist()
    k, v = randn(total, nkv, ps, hd, seed=seed + 1, dtype=dtype), randn(total, nkv, ps, hd, seed=seed + 2, dtype=dtype)
    whole = torch.full((len(reqs), max(-(-n // ps) for n, _ in reqs) + 1), -1, dtype=torch.int32)
    table = whole.clone()
    cu, it = [0], iter(perm)
    for r, (n, ql) in enumerate(reqs):
        for i in range(-(-n // ps)):
            whole[r, i] = table[r, i] = next(it)
            if window and i * ps >= keep and (i + 1) * ps - 1 < n - ql - window + 1:
                table[r, i] = -1
        cu.append(cu[-1] + ql)
    i32 = dict(dtype=torch.int32, device=DEV)
    return k, v, table.to(DEV), torch.tensor(cu, **i32), torch.tensor([n for n, _ in reqs], **i32), whole


CASES = [
    # nh, nkv, hd, page, window, keep, [(kv_len, q_len)]
    (4, 1, 128, 64, 150, 70, [(900, 900), (801, 1), (701, 203), (2, 2), (71, 1), (500, 1)]),
    (8, 8, 128, 64, 64, 64, [(400, 300), (665, 65), (129, 1), (128, 1)]),
    (2, 2, 128, 128, 40, 3, [(700, 260), (430, 130), (44, 4), (900, 1)]),
    (6, 3, 48, 16, 19, 33, [(100, 100), (175, 1), (38, 2), (212, 40), (60, 1)]),
    (8, 2, 64, 64, 70, 1, [(300, 300), (529, 1), (72, 1), (393, 66)]),
    (3, 1, 40, 16, 5, 7, [(90, 90), (77, 1), (300, 1), (260, 9)]),
    (12, 2, 128, 64, 100, 500, [(25, 1), (24, 1), (900, 1), (964, 5), (601, 1)]),
    (34, 1, 64, 64, 65, 129, [(700, 1), (300, 1), (450, 33)]),
    (4, 2, 96, 48, 21, 50, [(333, 1), (205, 60), (70, 1)]),
    (2, 1, 208, 16, 30, 20, [(200, 1), (155, 40)]),
    (4, 2, 32, 8, 1, 2, [(64, 64), (65, 1), (3, 1)]),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nh,nkv,hd,ps,window,keep,reqs", CASES)
@pytest.mark.parametrize("fast", [False, True])
def test_windowed_attention_with_kept_tokens(ops, slow_ops, dtype, nh, nkv, hd, ps, window, keep, reqs, fast):
    o, ref = (ops if fast else slow_ops), PlainOps()
    k, v, table, cu_q, kv_len, _ = paged(reqs, nkv, hd, ps, dtype, 21, window, keep)
    q = randn(int(cu_q[-1]), nh * hd, seed=22, dtype=dtype)
    scale = 1.5 / math.sqrt(hd)
    mq, mk, ns = max(ql for _, ql in reqs), max(n for n, _ in reqs), sum(1 for _, ql in reqs if ql == 1)
    args = (window, scale, nh, nkv, hd, mq, mk)
    got = o.attention(q, k, v, table, cu_q, kv_len, *args, ns, keep_first=keep)
    want = ref.attention(q.cpu(), k.cpu(), v.cpu(), table.cpu(), cu_q.cpu(), kv_len.cpu(), *args, keep_first=keep)
    o.check_errors()
    assert torch.allclose(got.float().cpu(), want.float(), **tol(dtype, 1e-4))
    # the single-token requests through the kernels for portions as well
    if fast and ns:
        again = o.attention(q, k, v, table, cu_q, kv_len, *args, 0, keep_first=keep)
        assert torch.allclose(again.float().cpu(), want.float(), **tol(dtype, 1e-4))
    # with other terms of a score beside it, and with more kept tokens than there are
    slopes = torch.linspace(0.01, 0.05, nh, device=DEV)
    sinks = torch.linspace(-1.0, 2.0, nh, device=DEV)
    for extra in ({"slopes": slopes, "sinks": sinks}, {"softcap": 2.0}):
        got = o.attention(q, k, v, table, cu_q, kv_len, *args, ns, keep_first=keep, **extra)
        cpu = {n: (x.cpu() if torch.is_tensor(x) else x) for n, x in extra.items()}
        want = ref.attention(q.cpu(), k.cpu(), v.cpu(), table.cpu(), cu_q.cpu(), kv_len.cpu(), *args, keep_first=keep, **cpu)
        assert torch.allclose(got.float().cpu(), want.float(), **tol(dtype, 1e-4))
    o.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("fast", [False, True])
@pytest.mark.parametrize("hd,ps,window,keep", [(128, 64, 64, 70), (128, 64, 193, 64), (64, 64, 100, 1), (48, 16, 33, 20), (40, 16, 9, 16)])
@pytest.mark.parametrize("q_len", [1, 2, 140])
def test_loud_keys_at_the_edges(ops, slow_ops, dtype, fast, hd, ps, window, keep, q_len):
    """One loud key at the window's first position, the one before it, the last kept position, the one behind it, and
    position 0: the last query returns its value where it is visible, the mean of the visible values where it is not."""
    o = ops if fast else slow_ops
    nh, nkv, n = 2, 1, 9 * ps + 5
    lo = n - window
    assert lo - 1 > keep
    k, v, table, cu_q, kv_len, whole = paged([(n, q_len)], nkv, hd, ps, dtype, 31, window, keep)
    q = randn(q_len, nh * hd, seed=32, dtype=dtype)
    q[-1, hd:] = q[-1, :hd]
    seen = list(range(keep)) + list(range(lo, n))
    vals = torch.stack([v[int(whole[0, i // ps]), 0, i % ps].float() for i in seen])
    for j in (lo, lo - 1, keep - 1, keep, 0):
        k.zero_()
        k[int(whole[0, j // ps]), 0, j % ps] = (q[-1, :hd].float() * 3.0).to(dtype)
        got = o.attention(q, k, v, table, cu_q, kv_len, window, 1.0 / math.sqrt(hd), nh, nkv, hd, q_len, n, int(q_len == 1),
                          keep_first=keep)
        o.check_errors()
        s = torch.zeros(len(seen), device=DEV)
        if j in seen:
            s[seen.index(j)] = float((q[-1, :hd].float() * k[int(whole[0, j // ps]), 0, j % ps].float()).sum()) / math.sqrt(hd)
        w = torch.softmax(s, 0)
        want = (w[:, None] * vals).sum(0)
        for h in range(nh):
            assert torch.allclose(got[-1, h * hd:(h + 1) * hd].float(), want, **tol(dtype, 1e-4)), j
        assert (float(w.max()) > 0.8) == (j in seen)


def test_a_missing_kept_page_is_reported(ops):
    for q_len in (1, 40):
        k, v, table, cu_q, kv_len, _ = paged([(500, q_len)], 1, 128, 64, torch.bfloat16, 3, 64, 10)
        table[0, 0] = -1
        q = randn(q_len, 128, seed=4, dtype=torch.bfloat16)
        ops.attention(q, k, v, table, cu_q, kv_len, 64, 0.1, 1, 1, 128, q_len, 500, int(q_len == 1), keep_first=10)
        torch.cuda.synchronize()
        with pytest.raises(Exception, match="no page"):
            ops.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("fast", [False, True])
@pytest.mark.parametrize("hd,ps,window,keep", [(128, 64, 150, 30), (128, 64, 0, 0), (64, 64, 80, 5), (96, 64, 50, 64), (48, 16, 20, 3),
                                               (32, 16, 0, 0), (176, 16, 33, 9)])
def test_two_maps_in_the_halves_of_a_head(ops, slow_ops, dtype, fast, hd, ps, window, keep):
    """Queries that are zero outside their half: whether a kernel is told so or not, and whatever the other half of the
    keys holds, the result is the plain one; the two maps differ."""
    o, ref = (ops if fast else slow_ops), PlainOps()
    nh, nkv = 8, 2
    reqs = [(400, 400), (333, 1), (290, 65), (7, 3)]
    k, v, table, cu_q, kv_len, _ = paged(reqs, nkv, hd, ps, dtype, 51, window, keep)
    T = int(cu_q[-1])
    q = randn(T, nh // 2, 2, hd, seed=52, std=1.4, dtype=dtype)
    q[:, :, 0, hd // 2:] = 0
    q[:, :, 1, :hd // 2] = 0
    q = q.reshape(T, nh * hd).contiguous()
    args = (window, 1.3 / math.sqrt(hd // 2), nh, nkv, hd, 400, 400)
    want = ref.attention(q.cpu(), k.cpu(), v.cpu(), table.cpu(), cu_q.cpu(), kv_len.cpu(), *args, keep_first=keep).float()
    for parts in (1, 2):
        got = o.attention(q, k, v, table, cu_q, kv_len, *args, 1, keep_first=keep, parts=parts)
        assert torch.allclose(got.float().cpu(), want, **tol(dtype, 1e-4))
    o.check_errors()
    m = want.reshape(T, nh // 2, 2, hd)
    assert float((m[:, :, 0] - m[:, :, 1]).abs().mean()) > 0.02


# ============================================================== the other kernels alone
SHAPES = [(6, 3, 20, 56, 64, 4), (5, 5, 7, 9, 16, 2), (8, 2, 64, 128, 128, 3), (3, 1, 9, 23, 32, 5), (2, 1, 48, 96, 96, 1),
          (4, 2, 100, 30, 208, 3), (2, 2, 13, 200, 208, 16), (16, 1, 32, 64, 64, 0), (1, 1, 128, 256, 256, 4)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv,D,taps", SHAPES)
@pytest.mark.parametrize("off", [0, 1])
def test_convolution_norm_and_write(ops, dtype, H, G, d, dv, D, taps, off):
    """Several requests with carried inputs that are larger than the new ones, single tokens beside portions, then the
    same tokens in other portions: queries, cache rows and carried inputs."""
    ref, ps = PlainOps(), 16
    C = 2 * (H + G) * d + G * dv
    w = randn(taps, C, seed=2) if taps else None
    qn, kn = randn(d, seed=3, std=0.3) + 1.0, randn(d, seed=4, std=0.3) - 1.5
    for lens in ([9, 1, 37, 2], [1, 1, 1], [200, 1, 3]):
        T = sum(lens)
        b = batch_of(lens, [3, 0, 4, 2][:len(lens)])
        proj = randn(T, C + 6 + off, seed=1)[:, off:]
        state = randn(5, max(taps - 1, 1), C, seed=5, std=3.0)[:, :max(taps - 1, 0)].contiguous()
        slots = torch.randperm(20 * ps, generator=torch.Generator().manual_seed(6))[:T].to(DEV, torch.int32)
        slots[T // 2] = -1
        caches = [torch.full((21, G, ps, D), 7.0, device=DEV, dtype=dtype) for _ in range(2)]
        wk, wv, ws = caches[0].cpu(), caches[1].cpu(), state.cpu()
        kc, vc, gs = caches[0].clone(), caches[1].clone(), state.clone()
        want = ref.map_norm_write(proj.cpu(), None if w is None else w.cpu(), ws, to_cpu(b), qn.cpu(), kn.cpu(), 1e-3, slots.cpu(), wk, wv,
                                  H, G, d, dv, D, dtype)
        got = ops.map_norm_write(proj, w, gs if taps > 1 else None, b, qn, kn, 1e-3, slots, kc, vc, H, G, d, dv, D, dtype)
        ops.check_errors()
        t = tol(dtype, 3e-5)
        assert torch.allclose(got.float().cpu(), want.float(), **t)
        assert torch.allclose(kc.float().cpu(), wk.float(), **t) and torch.allclose(vc.float().cpu(), wv.float(), **t)
        if taps > 1:
            assert torch.equal(gs.cpu(), ws)
            # request 0 alone in pieces: the same bits
            pieces = [n for n in (1, 2, 1, 5) if n <= lens[0]]
            at, ps_state = 0, state.clone()
            for n in pieces:
                if at + n > lens[0]:
                    break
                part = ops.map_norm_write(proj[at:at + n], w, ps_state, batch_of([n], [3]), qn, kn, 1e-3, slots[at:at + n].contiguous(),
                                          kc, vc, H, G, d, dv, D, dtype)
                assert torch.equal(part, got[at:at + n])
                at += n
    bad = slots.clone()
    bad[0] = 21 * ps
    ops.map_norm_write(proj, w, gs if taps > 1 else None, b, qn, kn, 1e-3, bad, kc, vc, H, G, d, dv, D, dtype)
    torch.cuda.synchronize()              # (the flag is set once the kernel has run)
    with pytest.raises(Exception, match="slot"):
        ops.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dv,D,off", [(6, 56, 64, 0), (3, 9, 16, 1), (16, 128, 128, 4), (5, 23, 32, 2), (2, 256, 256, 0), (1, 200, 208, 8),
                                        (7, 1, 16, 3), (4, 64, 64, 1)])
@pytest.mark.parametrize("T", [1, 37, 300])
def test_difference_norm_and_gate(ops, dtype, H, dv, D, off, T):
    """Two maps that nearly cancel in one head (the norm brings the rest up to size), what lies behind the values in a
    stored head is not read, and a negative lambda."""
    ref = PlainOps()
    o = randn(T, H, 2, D, seed=1, dtype=dtype)
    o[:, 0, 1] = o[:, 0, 0]
    o[..., dv:] = float("nan")
    o = o.reshape(T, 2 * H * D)
    gate = randn(T, H * dv + off + 3, seed=2, std=3.0)[:, off:off + H * dv]
    for lam in (0.9, 0.3, -0.4, 1.7):
        for g in (gate, None):
            got = ops.diff_norm_gate(o, g, H, dv, D, lam, 1e-4, 0.65)
            want = ref.diff_norm_gate(o.cpu(), None if g is None else g.cpu(), H, dv, D, lam, 1e-4, 0.65)
            assert got.dtype == dtype and torch.allclose(got.float().cpu(), want.float(), **tol(dtype, 2e-5, 1e-2))
    ops.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H", [(1, 192), (40, 63), (300, 2048), (3, 12288), (2, 12292), (1, 51204), (5, 1030)])
def test_embedding_positions_and_norm(ops, dtype, T, H):
    """One pass for the token's row, the position's row and their norm; a large eps, a scale, no positions; ids outside
    their tables are reported and nothing is read."""
    ref = PlainOps()
    table, pos = randn(50, H, seed=1, dtype=dtype), randn(33, H, seed=2, std=2.0, dtype=dtype)
    g = torch.Generator().manual_seed(3)
    ids, at = (torch.randint(0, n, (T,), generator=g).to(DEV, torch.int32) for n in (50, 33))
    w = randn(H, seed=4)
    for scale, added, eps in ((1.0, pos, 0.7), (1.0, None, 1e-6), (3.5, pos, 1e-5)):
        got = ops.embed_norm(ids, table, scale, added, at, w, eps)
        want = ref.embed_norm(ids.cpu(), table.cpu(), scale, None if added is None else added.cpu(), at.cpu(), w.cpu(), eps)
        assert got.dtype == torch.float32 and torch.allclose(got.cpu(), want, atol=1e-5, rtol=1e-5)
    ops.check_errors()
    for bad_ids, bad_at, what in ((ids + 50, at, "token id"), (ids, at + 33, "position")):
        ops.embed_norm(bad_ids, table, 1.0, pos, bad_at, w, 1e-5)
        torch.cuda.synchronize()
        with pytest.raises(Exception, match=what):
            ops.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,k,E,H", [(1, 1, 4, 192), (5, 3, 3, 62), (40, 2, 9, 1024), (300, 1, 16, 35), (64, 4, 8, 256)])
def test_weighted_rows_side_by_side(ops, dtype, T, k, E, H):
    """Each token's row times each of its weights, at the place its expert's group gives it; then combined unweighted."""
    ref = PlainOps()
    ids = torch.stack([torch.randperm(E, generator=torch.Generator().manual_seed(t))[:k] for t in range(T)]).to(DEV, torch.int32)
    offsets, rows, dest = ops.moe_permute(ids, E)
    h, wts = randn(T, H, seed=1, dtype=dtype), torch.rand(T, k, generator=torch.Generator().manual_seed(2)).to(DEV)
    got = ops.weigh_rows(h, wts, dest)
    assert torch.equal(got.cpu(), ref.weigh_rows(h.cpu(), wts.cpu(), dest.cpu()))
    for t in range(T):
        for j in range(k):
            assert torch.equal(got[dest[t, j].long()], (h[t].float() * wts[t, j]).to(dtype))
        if t > 20:
            break
    y, resid = randn(T * k, H, seed=3), randn(T, H, seed=4)
    want = resid.clone()
    for j in range(k):
        want += y[dest[:, j].long()]
    ops.moe_combine(y, dest, None, None, None, resid)
    ops.check_errors()
    assert torch.allclose(resid, want, atol=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,F,K", [(1, 320, 192), (8, 512, 1024), (40, 96, 256), (70, 200, 128), (300, 640, 512), (33, 15, 62), (5, 1, 8),
                                   (1000, 384, 320), (20, 33, 64)])
def test_clamped_gate(ops, slow_ops, dtype, M, F, K):
    """The clamped gate in the epilogue of every product kernel (streaming, small, warp-level, tcgen05, paired, FMA), with
    a good part of the sums beyond the limits, for two sets of constants."""
    a, g, u = randn(M, K, seed=1, dtype=dtype), randn(F, K, seed=2, std=K ** -0.5 * 2, dtype=dtype), randn(F, K, seed=3, std=K ** -0.5 * 2, dtype=dtype)
    w = torch.empty(2 * F, K, dtype=dtype, device=DEV)
    w[0::2], w[1::2] = g, u
    zg, zu = a.double() @ g.double().T, a.double() @ u.double().T
    for limit, alpha, shift in ((1.3, 1.702, 1.0), (0.4, 0.9, -0.5)):
        c = torch.tensor([limit, alpha, shift], device=DEV)
        z, y = zg.clamp(max=limit), zu.clamp(-limit, limit)
        want = z * torch.sigmoid(alpha * z) * (y + shift)
        for o in (ops, slow_ops):
            got = o.linear_clamped_glu(a, w, c)
            assert got.dtype == dtype and torch.allclose(got.double(), want, **tol(dtype, 2e-4, 3e-2))
    ops.check_errors()


def test_clamped_gate_far_out(ops):
    """Very negative gates give nothing (no overflow in the fast epilogues), very large ones the limit's value."""
    for M in (1, 32, 300):
        a = torch.zeros(M, 64, device=DEV, dtype=torch.bfloat16)
        a[:, 0] = 1.0
        w = torch.zeros(2 * 128, 64, device=DEV, dtype=torch.bfloat16)
        big = torch.linspace(-3000.0, 3000.0, 128).to(torch.bfloat16)
        w[0::2, 0], w[1::2, 0] = big.to(DEV), 9.0
        got = ops.linear_clamped_glu(a, w, torch.tensor([2.0, 1.702, 1.0], device=DEV)).float().cpu()
        z = big.double().clamp(max=2.0)
        want = (z * torch.sigmoid(1.702 * z) * 3.0).float().expand(M, 128)
        assert torch.allclose(got, want, rtol=1e-2, atol=1e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,k,H,ff", [(1, 8, 1, 192, 64), (7, 5, 5, 48, 22), (40, 16, 2, 256, 96), (300, 8, 3, 128, 80), (600, 4, 1, 320, 128)])
def test_experts_weighted_at_their_input(dtype, T, E, k, H, ff):
    """The part on its own: sigmoid scores as they are, in front of the expert."""
    from dlm_b200.engine.engine import make_runtime
    from dlm_b200.parts import PartSpec
    from dlm_b200.registry import build_part
    rt = make_runtime(dtype, DEV)
    part = build_part("ffn", PartSpec("moe_topk", {"hidden_size": H, "num_experts": E, "top_k": k, "expert_intermediate_size": ff,
                                                   "norm_topk_prob": False, "score": "sigmoid", "weigh": "input",
                                                   "names": {"router": "router", "gate": "e{e}.gate", "up": "e{e}.up", "down": "e{e}.down"}}))
    t = {s.name: randn(*s.shape, seed=i, std=2.0 / math.sqrt(s.shape[-1]), dtype=torch.bfloat16).cpu() for i, s in enumerate(part.param_specs())}
    part.load(t, rt)
    norm = build_part("norm", PartSpec("rmsnorm", {"size": H, "eps": 1e-5, "offset": 1.0}))
    norm.load({"weight": randn(H, seed=99, std=0.2).cpu()}, rt)
    x = randn(T, H, seed=100, std=2.0)
    resid = x.clone()
    part.forward(norm.forward(resid, rt), resid, SimpleNamespace(rt=rt), pre_norm=norm)
    rt.ops.check_errors()
    h = plain.model_norm(x.cpu().double(), norm.weight.cpu().double() - 1.0, 1e-5)
    p = lambda n: t[n].double()
    want = plain.weighted_input_experts(h, p, k, rounded=dtype == torch.bfloat16)
    z = torch.sort(h @ p("router").T, dim=-1, descending=True).values
    ok = (z[:, k - 1] - z[:, k] > 1e-3) if k < E else torch.ones(T, dtype=torch.bool)
    got = (resid - x).cpu().double()
    assert int(ok.sum()) > T // 2
    assert torch.allclose(got[ok], want[ok], **tol(dtype, 2e-4, 4e-2))


# ============================================================== the engine against the plain model
def gpu_engine(folder, dtype, **kw):
    from dlm_b200.engine import Engine
    args = dict(dtype=dtype, device=DEV, page_size=16, num_pages=64, max_requests=4)
    args.update(kw)
    return Engine.from_pretrained(folder, **args)


def check(got, ref, lim, dtype, what):
    """In bfloat16 a limit made from one rounded run is itself a noisy number: no row is beyond one and a half times its
    limit and at most one in fifty is beyond it.  At least four rows in five have a limit."""
    r = ratios(got, ref, lim)
    assert len(r) >= 0.8 * len(got), (what, len(r), len(got))
    print(f"{what} {dtype}: {len(r)} rows, worst error / limit {max(r):.2f}, {sum(x > 1 for x in r)} over")
    if dtype == "float32":
        assert max(r) < 1.0, (what, max(r))
    else:
        assert max(r) < 1.5 and sum(x > 1.0 for x in r) <= len(r) // 50, (what, max(r))


MIXERS = {
    "kept": attention(6, 3, 24, 40, 0.6, 0.3, 3, 13, 5),
    "no_kept": attention(2, 1, 12, 20, 0.7, 0.55, 4, 7),
    "no_window": attention(2, 2, 16, 30, 0.5, 0.2, 2),
    "no_convolution": attention(4, 1, 10, 18, 0.8, 0.4, None, 9, 20),
}


@pytest.mark.parametrize("kind", list(MIXERS))
@pytest.mark.parametrize("mlp", [None, dense(56, 1.1), moe(5, 2, 28)], ids=["none", "dense", "moe"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_each_layer_alone(kind, mlp, dtype, tmp_path):
    """A model of one layer: whole, token by token and in portions of two."""
    cfg = one_layer(layer(MIXERS[kind], mlp), width=72)
    oracle = plain.PlainGakenex(cfg, write_model(cfg, str(tmp_path / "m"), seed=11))
    reqs = clear_requests(oracle, [45])
    ref, lim = references(oracle, reqs, dtype)
    eng = gpu_engine(str(tmp_path / "m"), dtype)
    for steps in (cuttings.whole(reqs), cuttings.tail_decode(reqs, 44), cuttings.portions(reqs, sizes=(2,))):
        check(cuttings.run_trace(eng, steps), ref, lim, dtype, kind)


def test_residual_after_every_layer(folders):
    folder, oracle = folders["A"]
    toks = clear_requests(oracle, [50], seed=3)["r0"]
    _, after = oracle.forward(toks, trace=True)
    eng = gpu_engine(folder, "float32")
    seen = []
    eng.model.after_layer = lambda call, x: seen.append(x.detach().double().cpu())
    slot = eng.cache.open()
    eng.step([(slot, toks, [])])
    eng.cache.close(slot)
    assert len(seen) == after.shape[0]
    for i, x in enumerate(seen):
        assert float((x - after[i]).abs().max() / after[i].abs().max()) < 5e-5, i


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_every_cutting_matches_the_plain_model(name, dtype, folders):
    """Prefill against decoding token by token, portions down to two tokens, unequal requests batched against each
    alone, requests many windows and pages long in prompts and in decoding."""
    folder, oracle = folders[name]
    reqs = clear_requests(oracle, [1, 2, 23, 150, 410])
    ref, lim = references(oracle, reqs, dtype)
    page = 64 if name == "C" else 16
    eng = gpu_engine(folder, dtype, page_size=page, num_pages=1024 // page)
    mixed, _ = cuttings.mixed(reqs, max_live=4, seed=1, decode_tail=70 if name == "A" else 24)
    for what, steps in (("whole", cuttings.whole(reqs)), ("decode", cuttings.tail_decode(reqs, 300 if name == "C" else 120)),
                        ("portions", cuttings.portions(reqs)), ("mixed", mixed)):
        got = cuttings.run_trace(eng, steps)
        assert len(got) == sum(len(t) for t in reqs.values())
        check(got, ref, lim, dtype, f"{name} {what}")
    assert all(p.used_pages == 0 for p in eng.cache.stats())


def test_cuttings_agree_to_the_last_bit_in_32_bit(folders):
    """In 32-bit every kernel adds in an order of its own that does not depend on the cut: logits are equal bit for
    bit whether a request came whole, token by token, or beside others."""
    folder, _ = folders["A"]
    V = CONFIGS["A"]["vocab"]
    reqs = {f"r{i}": tokens(30 + i, n, V) for i, n in enumerate([5, 130, 33])}
    eng = gpu_engine(folder, "float32")
    base = cuttings.run_trace(eng, cuttings.whole(reqs))
    mixed, _ = cuttings.mixed(reqs, max_live=3, seed=4)
    for steps in (cuttings.tail_decode(reqs, 30), cuttings.portions(reqs, sizes=(2, 3)), mixed):
        got = cuttings.run_trace(eng, steps)
        assert all(torch.equal(got[k], base[k]) for k in base)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "D"])
def test_slots_and_pages_used_again(name, dtype, folders):
    """Eight requests through three slots and a pool that holds only what is live."""
    folder, oracle = folders[name]
    reqs = clear_requests(oracle, [70, 33, 129, 16, 90, 7, 64, 65], seed=20)
    steps, _ = cuttings.mixed(reqs, max_live=3, seed=2)
    eng = gpu_engine(folder, dtype, num_pages=cuttings.peak_tokens(steps) // 16, max_requests=3)
    got = cuttings.run_trace(eng, steps)
    ref, lim = references(oracle, reqs, dtype)
    check(got, ref, lim, dtype, name)
    assert all(s.used_pages == 0 for s in eng.cache.stats())


@pytest.mark.parametrize("name,dtype", [("B", "float32"), ("A", "float32"), ("C", "bfloat16"), ("D", "bfloat16")])
def test_long_greedy_generation_through_scheduler_and_graphs(name, dtype, folders):
    """Engine.generate's parts: prompts in portions under a token budget, then 200 decode steps replayed from graphs,
    states, windows and kept tokens carried all the way.  Every produced token is the plain model's choice wherever that
    is clear (and no choice of experts in front of it was close), and in 32-bit the logits of the last step agree."""
    folder, oracle = folders[name]
    V = CONFIGS[name]["vocab"]
    prompts = list(clear_requests(oracle, [70, 3, 129], seed=60).values())
    page = 64 if name == "C" else 16
    eng = gpu_engine(folder, dtype, page_size=page, num_pages=2048 // page, max_step_tokens=48, max_context=512)
    assert eng.use_graphs
    news = [200, 40, 90]
    ids = [eng.submit(p, max_new_tokens=n) for p, n in zip(prompts, news)]
    last = {}
    while eng.scheduler.has_work():
        produced = eng.run_step()
        if len(produced) == 1 and eng.last_logits.shape[0] == 1:
            last["row"] = eng.last_logits[0].float().cpu().clone()
    outs = [eng.result(i) for i in ids]
    assert eng.graphs_recorded > 0 and [len(o) for o in outs] == news
    seqs = {str(i): p + out[:-1] for i, (p, out) in enumerate(zip(prompts, outs))}
    ref, lim = references(oracle, seqs, dtype)
    clear = 0
    for i, (p, out) in enumerate(zip(prompts, outs)):
        for j, tok in enumerate(out):
            at = len(p) - 1 + j
            row = ref[str(i)][at]
            top2 = torch.topk(row, 2).values
            spread = float((row - row.mean()).pow(2).mean().sqrt())
            if float(top2[0] - top2[1]) > 4 * float(lim[str(i)][at]) * spread:
                assert int(torch.argmax(row)) == tok, (name, dtype, i, j)
                clear += 1
    print(f"{name} {dtype}: {clear} of {sum(news)} tokens were clear choices")
    assert clear >= (sum(news) // 2 if dtype == "float32" else 5)
    if dtype == "float32":
        assert float(row_error(last["row"], ref["0"][-1])) < 1e-4


def test_command_line_with_random_weights(tmp_path):
    """`dlm-b200 generate --random CONFIG.json --save-random DIR`: the architecture is found through the registry, the
    weights are drawn and written, and the ids printed are the plain model's greedy choices on that folder."""
    import ast
    import json
    import os
    import subprocess
    import sys
    from plain_zesapel import read_safetensors            # the file format alone, nothing of the package
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg_path, folder = str(tmp_path / "config.json"), str(tmp_path / "model")
    with open(cfg_path, "w") as f:
        json.dump(CONFIGS["A"], f)
    prompts = [[5, 6, 7, 100, 3], [9]]
    cmd = [sys.executable, os.path.join(root, "bin", "dlm-b200"), "generate", "--random", cfg_path, "--seed", "3",
           "--save-random", folder, "--max-new-tokens", "6", "--dtype", "float32"]
    for p in prompts:
        cmd += ["--prompt", ",".join(str(t) for t in p)]
    out = subprocess.run(cmd, capture_output=True, text=True, timeout=900)
    assert out.returncode == 0, out.stderr[-2000:]
    lines = [ln for ln in out.stdout.splitlines() if ln.startswith("generated ids:")]
    assert len(lines) == len(prompts)
    oracle = plain.PlainGakenex(CONFIGS["A"], read_safetensors(os.path.join(folder, "model.safetensors")))
    for p, ln in zip(prompts, lines):
        ids = ast.literal_eval(ln.split(":", 1)[1].strip())
        assert len(ids) == 6
        seq = list(p)
        for tok in ids:
            row = oracle.forward(seq)[-1]
            top2 = torch.topk(row, 2).values
            if float(top2[0] - top2[1]) > 1e-3 * float((row - row.mean()).pow(2).mean().sqrt()):
                assert int(torch.argmax(row)) == tok
            seq.append(tok)


MID = model(1000, 320, [
    layer(attention(10, 5, 40, 80, 0.35, 0.3, 4, 130, 40), dense(512, 2.2)),
    layer(attention(8, 2, 64, 112, 0.25, 0.5, 3, 200, 65), moe(12, 3, 160)),
    layer(attention(16, 8, 24, 64, 0.45, 0.15, 2, 64, 128)),
    layer(attention(6, 1, 64, 128, 0.25, 0.6, 4), moe(24, 1, 96))], eps=1e-6, cap=15.0, positions=800)

ODD = model(1001, 201, [
    layer(attention(1, 1, 128, 256, 0.15, 0.4, 16, 33, 70), dense(7, 0.5)),
    layer(attention(12, 4, 3, 2, 1.4, 0.25, 7, 65, 64), moe(2, 2, 5)),
    layer(attention(2, 2, 70, 9, 0.2, 0.7, 3, 2, 1), moe(33, 1, 17)),
    layer(attention(34, 2, 8, 16, 0.7, 0.35, None, 100, 3), dense(88, 8.0))], eps=1e-4, cap=None, positions=300)


@pytest.mark.parametrize("cfg,lens,tail", [(MID, [37, 130, 420], 140), (ODD, [3, 70, 260], 60)], ids=["wider", "unusual"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_other_sizes_with_a_long_request(cfg, lens, tail, dtype, tmp_path):
    """wider: sizes between the tiny configurations and a real model's (products large enough for the tensor-core
    kernels, pages of 64).  unusual: keys and values as wide as the kernels take, wider than any tensor-core kernel, and
    tiny ones, sixteen taps, more query heads on a key than a tile has rows, a width that is no multiple of anything."""
    oracle = plain.PlainGakenex(cfg, write_model(cfg, str(tmp_path / "m"), seed=5))
    reqs = clear_requests(oracle, lens)
    ref, lim = references(oracle, reqs, dtype)
    eng = gpu_engine(str(tmp_path / "m"), dtype, page_size=64, num_pages=32)
    mixed, _ = cuttings.mixed(reqs, max_live=3, seed=2, decode_tail=40)
    for what, steps in (("whole", cuttings.whole(reqs)), ("decode", cuttings.tail_decode(reqs, tail)),
                        ("portions", cuttings.portions(reqs)), ("mixed", mixed)):
        check(cuttings.run_trace(eng, steps), ref, lim, dtype, what)
