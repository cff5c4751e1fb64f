"""Zepilorn on the GPU.  Kernels alone against their plain PyTorch statements, with inputs made so that a fault shows
(rows whose mean is far from zero, a stretched rotation in front of a norm, one loud key at either side of a window's
edge, quiet keys of which the silent sink takes its share, something written into the recurrent state hundreds of
tokens ago); then the engine against the plain model: single layers of every kind, four configurations of unlike sizes
under every cutting in both precisions, layers that read an earlier layer's keys and look further back than it, slots
and pages that are used again, long greedy decoding through the scheduler and the replayed graphs, the command line."""
import math
from types import SimpleNamespace

import pytest
import torch

import cuttings
import plain_zepilorn as plain
from plain_ops import PlainOps
from zepilorn_models import (CONFIGS, TOL, attention, latent, layer, linear, model, one_layer, ratios, references, row_error,
                             tokens, write_model, yarn)

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
    base = tmp_path_factory.mktemp("zepilorn_gpu")
    out = {}
    for name, cfg in CONFIGS.items():
        folder = str(base / name)
        out[name] = (folder, plain.PlainZepilorn(cfg, write_model(cfg, folder, seed=ord(name))))
    return out


def batch_of(lengths, slots, starts=None):
    """The fields of a step the kernels read, for requests that bring ``lengths`` tokens from ``starts`` on."""
    starts = starts or [0] * len(lengths)
    cu = [0]
    for n in lengths:
        cu.append(cu[-1] + n)
    i32 = dict(dtype=torch.int32, device=DEV)
    return SimpleNamespace(
        num_requests=len(lengths), cu_q=torch.tensor(cu, **i32), state_slot=torch.tensor(slots, **i32),
        token_req=torch.tensor([r for r, n in enumerate(lengths) for _ in range(n)], **i32),
        positions=torch.tensor([s + i for s, n in zip(starts, lengths) for i in range(n)], **i32))


def to_cpu(b):
    return SimpleNamespace(**{k: (v.cpu() if torch.is_tensor(v) else v) for k, v in vars(b).items()})


def randn(*shape, seed=0, std=1.0, dtype=torch.float32):
    return (std * torch.randn(*shape, generator=torch.Generator().manual_seed(seed))).to(DEV, dtype)


def tol(dtype, f32=2e-5, bf16=2e-2):
    return dict(atol=f32, rtol=f32) if dtype == torch.float32 else dict(atol=bf16, rtol=bf16)


# ============================================================== kernels alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W", [(1, 48), (37, 62), (300, 1024), (5, 2051), (3, 4096), (2, 12288), (4, 192), (7, 3)])
def test_norms_on_outputs(ops, dtype, T, W):
    """The centred norm (of chosen rows as well), and the closing step of a sublayer: norm, add, rounded copy, rows
    cleared; centred and not.  The rows' means are many times their spread: a variance made of squares would be off."""
    ref = PlainOps()
    x = randn(T, W, seed=1, std=2.0) + 50.0
    w, b = randn(W, seed=2, std=0.3) + 1.0, randn(W, seed=3, std=0.3)
    got = ops.layer_norm(x, w, b, 1e-5, dtype)
    want = ref.layer_norm(x.cpu().double(), w.cpu().double(), b.cpu().double(), 1e-5, torch.float64)
    assert got.dtype == dtype and torch.allclose(got.double().cpu(), want, **tol(dtype, 2e-4))
    rows = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32, device=DEV)
    assert torch.equal(ops.layer_norm(x, w, b, 1e-5, dtype, rows), got[rows.long()])
    for bias in (b, None):
        resid, y = randn(T, W, seed=4, std=3.0), x.clone()
        want = resid.cpu().double()
        ref.post_norm_add(want, x.cpu().double(), w.cpu().double(), None if bias is None else b.cpu().double(), 1e-5, torch.float64)
        for clear in (False, True):
            r2, y2 = resid.clone(), y.clone()
            out = ops.post_norm_add(r2, y2, w, bias, 1e-5, dtype, clear=clear)
            assert torch.allclose(r2.double().cpu(), want, atol=2e-4, rtol=2e-4)
            assert (out is r2) if dtype == torch.float32 else torch.equal(out, r2.to(dtype))
            assert torch.equal(y2, torch.zeros_like(y2) if clear else y)
    ops.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("act", ["gelu_tanh", "silu"])
@pytest.mark.parametrize("M,F,K", [(1, 320, 192), (8, 512, 1024), (40, 96, 256), (70, 200, 128), (300, 640, 512), (33, 15, 62),
                                   (5, 1, 8), (1000, 384, 320)])
def test_gated_product(ops, slow_ops, dtype, act, M, F, K):
    """act(gate) * up in the epilogue of every product kernel (streaming, small, warp-level, tcgen05, paired, FMA)."""
    a, g, u = randn(M, K, seed=1, dtype=dtype), randn(F, K, seed=2, std=K ** -0.5 * 2, dtype=dtype), randn(F, K, seed=3, std=K ** -0.5, dtype=dtype)
    w = torch.empty(2 * F, K, dtype=dtype, device=DEV)
    w[0::2], w[1::2] = g, u
    z = a.double() @ g.double().T
    z = torch.nn.functional.gelu(z, approximate="tanh") if act == "gelu_tanh" else torch.nn.functional.silu(z)
    want = z * (a.double() @ u.double().T)
    for o in (ops, slow_ops):
        got = o.linear_glu(a, w, act)
        assert got.dtype == dtype and torch.allclose(got.double(), want, **tol(dtype, 2e-4, 3e-2))
    ops.check_errors()


def test_gated_product_saturates(ops):
    """Far from zero the tanh form is the input itself or nothing, without overflow, in the fast epilogues as well."""
    for M in (1, 32, 300):
        a = torch.zeros(M, 64, device=DEV, dtype=torch.bfloat16)
        a[:, 0] = 1.0
        w = torch.zeros(2 * 128, 64, device=DEV, dtype=torch.bfloat16)
        big = torch.linspace(-3000.0, 3000.0, 128).to(torch.bfloat16)
        w[0::2, 0], w[1::2, 0] = big.to(DEV), 1.0
        got = ops.linear_glu(a, w, "gelu_tanh").float().cpu()
        assert torch.allclose(got, torch.nn.functional.gelu(big.float(), approximate="tanh").expand(M, 128), rtol=1e-2, atol=1e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nh,nkv,d,dv,D,rot,interleaved", [(6, 3, 24, 40, 48, 16, False), (4, 4, 10, 6, 16, 10, False),
                                                           (8, 2, 128, 128, 128, 64, False), (3, 1, 33, 20, 48, 8, True),
                                                           (5, 5, 12, 20, 32, 0, False), (2, 1, 96, 64, 96, 96, True)])
def test_rotation_with_an_amplitude_then_the_norm(ops, dtype, nh, nkv, d, dv, D, rot, interleaved):
    """The rotation stretches part of every head and the norm behind it measures the stretched head; with a small head
    and a large eps, a norm in front of the rotation, or one that forgot the amplitude, is far off."""
    ref = PlainOps()
    T, ps = 23, 16
    b = batch_of([T], [0], starts=[900])
    proj = randn(T, (nh + nkv) * d + nkv * dv + 5, seed=1, std=0.3)[:, 2:-3]
    inv_freq = (1000.0 ** (-torch.arange(0, max(rot, 2), 2).float() / max(rot, 2))).to(DEV)
    slots = torch.tensor([2 * ps + 5 + i if i < 11 else (i - 11 if i < 20 else -1) for i in range(T)], dtype=torch.int32, device=DEV)
    kc, vc = (torch.zeros(3, nkv, ps, D, device=DEV, dtype=dtype) for _ in range(2))
    wk, wv = kc.clone().cpu(), vc.clone().cpu()
    args = (1.7, True)
    want = ref.head_norm_rope_write(proj.cpu(), b.positions.cpu(), None, None, 0.05, inv_freq.cpu(), rot, interleaved, slots.cpu(),
                                    wk, wv, nh, nkv, d, dv, D, dtype, *args)
    got = ops.head_norm_rope_write(proj, b.positions, None, None, 0.05, inv_freq, rot, interleaved, slots, kc, vc, nh, nkv, d, dv,
                                   D, dtype, *args)
    t = tol(dtype, 3e-4)
    assert torch.allclose(got.float().cpu(), want.float(), **t)
    assert torch.allclose(kc.float().cpu(), wk.float(), **t) and torch.allclose(vc.float().cpu(), wv.float(), **t)
    # queries alone: the same bits, and nothing is written
    before = kc.clone(), vc.clone()
    only_q = ops.head_norm_rope_write(proj[:, :nh * d].contiguous(), b.positions, None, None, 0.05, inv_freq, rot, interleaved,
                                      None, kc, vc, nh, nkv, d, dv, D, dtype, *args)
    assert torch.equal(only_q, got) and torch.equal(kc, before[0]) and torch.equal(vc, before[1])
    if rot:
        for other in ((1.0, True), (1.7, False)):
            off = ref.head_norm_rope_write(proj.cpu(), b.positions.cpu(), None, None, 0.05, inv_freq.cpu(), rot, interleaved,
                                           slots.cpu(), wk.clone(), wv.clone(), nh, nkv, d, dv, D, dtype, *other)
            assert not torch.allclose(off.float(), want.float(), rtol=0.1, atol=0.1)
    ops.check_errors()


@pytest.mark.parametrize("heads,dk,dv", [(3, 10, 14), (1, 9, 5), (4, 32, 64), (2, 64, 128), (2, 40, 56), (1, 200, 24), (5, 3, 3)])
def test_scan_with_activated_inputs(ops, heads, dk, dv):
    """silu on values, keys and queries inside the scan (few tokens) and in front of it (many) against the plain
    statement, several requests with states that are not zero; cutting the tokens anywhere gives the same bits."""
    ref = PlainOps()
    decay = torch.linspace(0.0, 1.0, heads + 1)[1:].to(DEV)
    for lens in ([9, 1, 37], [90, 2, 41]):
        T = sum(lens)
        x = randn(T, heads * dv + 2 * heads * dk + 3, seed=1)[:, 1:-2]
        S = randn(5, heads, dk, dv, seed=4, std=0.2)
        b = batch_of(lens, [3, 0, 4])
        wS, gS = S.clone().cpu(), S.clone()
        call = lambda o, xx, st, bb, dd: o.ssm_scan(xx, None, None, None, None, st, bb, heads, dv, dk, heads, fixed_decay=dd,
                                                    silu_inputs=True)
        want = call(ref, x.cpu(), wS, to_cpu(b), decay.cpu())
        got = call(ops, x.clone(), gS, b, decay)
        ops.check_errors()
        assert torch.allclose(got.cpu(), want, atol=3e-4, rtol=3e-4) and torch.allclose(gS.cpu(), wS, atol=3e-4, rtol=3e-4)
        assert torch.equal(gS[1], S[1]) and torch.equal(gS[2], S[2])                          # slots not named
        # request 0 alone in pieces
        pS, outs, at = S.clone(), [], 0
        for c in (1, 2, 5, lens[0] - 8):
            outs.append(call(ops, x[at:at + c].clone(), pS, batch_of([c], [3]), decay))
            at += c
        assert torch.equal(torch.cat(outs), got[:lens[0]]) and torch.equal(pS[3], gS[3])


def test_scan_remembers_a_far_write(ops):
    """Decay 1: what token 0 wrote is read back exactly 400 tokens later; decay 0: only the token's own write is there."""
    dk, dv, T = 24, 20, 401
    x = torch.full((T, 2 * dv + 4 * dk), -1e4, device=DEV)            # silu of it is 0
    v, k, q = x[:, :2 * dv].view(T, 2, dv), x[:, 2 * dv:2 * dv + 2 * dk].view(T, 2, dk), x[:, 2 * dv + 2 * dk:].view(T, 2, dk)
    v[0], k[0, :, 5], q[T - 1, :, 5] = 30.0, 30.0, 30.0               # silu(30) is 30
    v[T - 1], k[T - 1, :, 5] = 40.0, 40.0
    S = torch.zeros(2, 2, dk, dv, device=DEV)
    decay = torch.tensor([1.0, 0.0], device=DEV)
    o = ops.ssm_scan(x, None, None, None, None, S, batch_of([T], [1]), 2, dv, dk, 2, fixed_decay=decay, silu_inputs=True)
    assert torch.allclose(o[T - 1, :dv], torch.full((dv,), 30.0 * (30 * 30 + 40 * 40.0), device=DEV), rtol=1e-5)
    assert torch.allclose(o[T - 1, dv:], torch.full((dv,), 30.0 * 40 * 40.0, device=DEV), rtol=1e-5)
    assert float(o[1:T - 1].abs().max()) == 0.0 and float(S[0].abs().max()) == 0.0
    ops.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mode", ["sigmoid_after", "silu_after"])
@pytest.mark.parametrize("groups,gs,off", [(1, 42, 3), (1, 512, 0), (1, 2048, 4), (2, 1000, 0), (1, 2048, 1), (1, 9000, 0), (1, 8192, 8)])
def test_one_norm_over_all_heads_with_a_gate(ops, dtype, mode, groups, gs, off):
    ref = PlainOps()
    T = 7
    y = randn(T, groups * gs, seed=1, std=4.0)
    gate = randn(T, groups * gs + off + 4, seed=2, std=2.0)[:, off:off + groups * gs]
    for w in (randn(groups * gs, seed=3, std=0.2) + 1.0, None):
        got = ops.gated_rmsnorm(y, gate, w, groups, 1e-5, mode, dtype)
        want = ref.gated_rmsnorm(y.cpu(), gate.cpu(), None if w is None else w.cpu(), groups, 1e-5, mode, dtype)
        assert torch.allclose(got.float().cpu(), want.float(), **tol(dtype, 1e-5))
    ops.check_errors()


# -------------------------------------------------------------- attention over a window with a silent sink
def paged(reqs, nkv, hd, ps, dtype, seed):
    """reqs: [(kv_len, q_len)].  Pages scattered over the pool.  Returns k, v, table, cu_q, kv_len."""
    total = sum(-(-n // ps) for n, _ in reqs) + 3
    perm = torch.randperm(total, generator=torch.Generator().manual_seed(seed)).tolist()
    k, v = randn(total, nkv, ps, hd, seed=seed + 1, dtype=dtype), randn(total, nkv, ps, hd, seed=seed + 2, dtype=dtype)
    table = torch.full((len(reqs), max(-(-n // ps) for n, _ in reqs) + 1), -1, dtype=torch.int32)
    cu, it = [0], iter(perm)
    for r, (n, ql) in enumerate(reqs):
        for i in range(-(-n // ps)):
            table[r, i] = next(it)
        cu.append(cu[-1] + ql)
    i32 = dict(dtype=torch.int32, device=DEV)
    return k, v, table.to(DEV), torch.tensor(cu, **i32), torch.tensor([n for n, _ in reqs], **i32)


CASES = [
    # nh, nkv, hd, page, window, [(kv_len, q_len)]
    (4, 1, 128, 64, 150, [(700, 700), (401, 1), (601, 203), (2, 2)]),
    (8, 8, 128, 64, 64, [(300, 300), (65, 65)]),
    (2, 2, 128, 128, 0, [(500, 260), (130, 130)]),
    (6, 3, 48, 16, 19, [(100, 100), (75, 1), (38, 2), (112, 40)]),
    (8, 2, 64, 64, 70, [(300, 300), (129, 1), (128, 1), (193, 66)]),
    (3, 1, 40, 16, 1, [(90, 90), (77, 1)]),
    (12, 2, 128, 64, 100, [(25, 1), (24, 1), (500, 1), (164, 1)]),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nh,nkv,hd,ps,window,reqs", CASES)
@pytest.mark.parametrize("fast", [False, True])
@pytest.mark.parametrize("sink", [0.0, 3.0, -60.0])
def test_windowed_attention_with_a_constant_sink(ops, slow_ops, dtype, nh, nkv, hd, ps, window, reqs, fast, sink):
    o, ref = (ops if fast else slow_ops), PlainOps()
    k, v, table, cu_q, kv_len = paged(reqs, nkv, hd, ps, dtype, 21)
    q = randn(int(cu_q[-1]), nh * hd, seed=22, dtype=dtype)
    sinks = torch.full((nh,), sink, device=DEV)
    scale = 1.5 / math.sqrt(hd)
    mq, mk, ns = max(ql for _, ql in reqs), max(n for n, _ in reqs), sum(1 for _, ql in reqs if ql == 1)
    got = o.attention(q, k, v, table, cu_q, kv_len, window, scale, nh, nkv, hd, mq, mk, ns, sinks=sinks)
    want = ref.attention(q.cpu(), k.cpu(), v.cpu(), table.cpu(), cu_q.cpu(), kv_len.cpu(), window, scale, nh, nkv, hd, mq, mk,
                         sinks=sinks.cpu())
    o.check_errors()
    assert torch.allclose(got.float().cpu(), want.float(), **tol(dtype, 1e-4))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("fast", [False, True])
@pytest.mark.parametrize("hd,ps,window", [(128, 64, 64), (128, 64, 193), (64, 64, 100), (48, 16, 33)])
@pytest.mark.parametrize("q_len", [1, 2, 140])
def test_the_key_at_the_windows_edge(ops, slow_ops, dtype, fast, hd, ps, window, q_len):
    """One loud key just inside the last query's window is what that query returns; one token further back it is not
    seen at all, and with every other key silent the output is the mean of the visible values times n / (n + 1)."""
    o = ops if fast else slow_ops
    nh, nkv, n = 2, 1, 6 * ps + 5
    k, v, table, cu_q, kv_len = paged([(n, q_len)], nkv, hd, ps, dtype, 31)
    q = randn(q_len, nh * hd, seed=32, dtype=dtype)
    q[-1, hd:] = q[-1, :hd]
    scale = 1.0 / math.sqrt(hd)
    zero = torch.zeros(nh, device=DEV)
    for inside in (True, False):
        j = n - 1 - (window - 1 if inside else window)
        k.zero_()
        k[int(table[0, j // ps]), 0, j % ps] = (q[-1, :hd].float() * 3.0).to(dtype)
        got = o.attention(q, k, v, table, cu_q, kv_len, window, scale, nh, nkv, hd, q_len, n, int(q_len == 1), sinks=zero)
        o.check_errors()
        vals = torch.stack([v[int(table[0, i // ps]), 0, i % ps].float() for i in range(n - window, n)])
        s = torch.zeros(window, device=DEV)
        if inside:
            s[0] = float((q[-1, :hd].float() * k[int(table[0, j // ps]), 0, j % ps].float()).sum()) * scale
        top = max(float(s.max()), 0.0)
        w = torch.exp(s - top)
        want = (w[:, None] * vals).sum(0) / (w.sum() + math.exp(-top))
        for h in range(nh):
            assert torch.allclose(got[-1, h * hd:(h + 1) * hd].float(), want, **tol(dtype, 1e-4))
        assert (float(s[0]) > 8.0) == inside


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("fast", [False, True])
@pytest.mark.parametrize("H,rank,ps,window", [(8, 128, 64, 90), (3, 28, 16, 33), (5, 256, 64, 64), (2, 72, 16, 0), (20, 128, 16, 1)])
@pytest.mark.parametrize("lens,starts", [([1], [200]), ([60, 1, 2], [70, 150, 40])])
def test_latent_attention_without_positions(ops, slow_ops, dtype, fast, H, rank, ps, window, lens, starts):
    """No rotated part, no sink: against the plain statement, with one latent just inside and one just outside the last
    query's window made loud."""
    o, ref = (ops if fast else slow_ops), PlainOps()
    reqs = [(s + n, n) for s, n in zip(starts, lens)]
    _, _, table, _, _ = paged(reqs, 1, rank, ps, dtype, 41)
    cache = randn(int(table.max()) + 2, 1, ps, rank, seed=42, std=0.3, dtype=dtype)
    b = batch_of(lens, list(range(len(lens))), starts)
    b.max_kv_len = max(n for n, _ in reqs)
    T = sum(lens)
    q_lat, q_rot = randn(H, T, rank, seed=43), torch.empty(T, H, 0, device=DEV)
    if window:
        for r, (n, _) in enumerate(reqs):
            last = int(b.cu_q[r + 1]) - 1
            for j, boost in ((n - window, 6.0), (n - window - 1, 6.0)):
                if j >= 0:
                    cache[int(table[r, j // ps]), 0, j % ps] = (q_lat[:, last].mean(0) * boost).to(dtype)
    got = o.latent_attention(q_lat, q_rot, None, cache, table, b, H, 0, rank, window, 0.2)
    want = ref.latent_attention(q_lat.cpu(), q_rot.cpu(), None, cache.cpu(), table.cpu(), to_cpu(b), H, 0, rank, window, 0.2)
    o.check_errors()
    assert torch.allclose(got.float().cpu(), want.float(), **tol(dtype, 1e-4, 3e-2))


# ============================================================== the engine against the plain model
def gpu_engine(folder, dtype, **kw):
    from dlm_b200.engine import Engine
    args = dict(dtype=dtype, device=DEV, page_size=16, num_pages=64, max_requests=4)
    args.update(kw)
    return Engine.from_pretrained(folder, **args)


def check(got, ref, lim, dtype, what):
    """In bfloat16 a limit made from one rounded run is itself a noisy number: no row is beyond one and a half times its
    limit and at most one in fifty is beyond it."""
    r = ratios(got, ref, lim)
    print(f"{what} {dtype}: {len(r)} rows, worst error / limit {max(r):.2f}, {sum(x > 1 for x in r)} over")
    if dtype == "float32":
        assert max(r) < 1.0, (what, max(r))
    else:
        assert max(r) < 1.5 and sum(x > 1.0 for x in r) <= len(r) // 50, (what, max(r))


MIXERS = {
    "attention": attention(6, 3, 24, 40, 1.2, 13, 5000.0, 16, yarn(6.0, 64, 8.0, 0.5)),
    "attention_no_rotation": attention(2, 1, 12, 20, 1.5, 7),
    "attention_no_window": attention(2, 2, 16, 8, 1.0, None, 100.0),
    "latent": latent(3, 20, 12, 28, 0.3, 11),
    "linear": linear(10, 14, [0.3, 0.9, 0.999]),
}


@pytest.mark.parametrize("kind", list(MIXERS))
@pytest.mark.parametrize("ff", [None, 56])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_each_mixer_alone(kind, ff, dtype, tmp_path):
    """A model of one layer: the mixer (and the feed-forward) alone, whole, token by token and in portions of two."""
    cfg = one_layer(layer(MIXERS[kind], ff), width=72)
    oracle = plain.PlainZepilorn(cfg, write_model(cfg, str(tmp_path / "m"), seed=11))
    reqs = {"a": tokens(1, 45, cfg["vocab"])}
    ref, lim = references(oracle, reqs, dtype)
    eng = gpu_engine(str(tmp_path / "m"), dtype)
    for steps in (cuttings.whole(reqs), cuttings.tail_decode(reqs, 44), cuttings.portions(reqs, sizes=(2,))):
        check(cuttings.run_trace(eng, steps), ref, lim, dtype, kind)


def test_residual_after_every_layer(folders):
    folder, oracle = folders["A"]
    toks = tokens(3, 50, CONFIGS["A"]["vocab"])
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
    V = CONFIGS[name]["vocab"]
    reqs = {f"r{i}": tokens(i, n, V) for i, n in enumerate([1, 2, 23, 150, 410])}
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
    reqs = {f"r{i}": tokens(30 + i, n, V) for i, n in enumerate([5, 90, 33])}
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
    V = CONFIGS[name]["vocab"]
    reqs = {f"q{i}": tokens(20 + i, n, V) for i, n in enumerate([70, 33, 129, 16, 90, 7, 64, 65])}
    steps, _ = cuttings.mixed(reqs, max_live=3, seed=2)
    eng = gpu_engine(folder, dtype, num_pages=cuttings.peak_tokens(steps) // 16, max_requests=3)
    got = cuttings.run_trace(eng, steps)
    ref, lim = references(oracle, reqs, dtype)
    check(got, ref, lim, dtype, name)
    assert all(s.used_pages == 0 for s in eng.cache.stats())


@pytest.mark.parametrize("name,dtype", [("B", "float32"), ("A", "float32"), ("C", "bfloat16")])
def test_long_greedy_generation_through_scheduler_and_graphs(name, dtype, folders):
    """Engine.generate's parts: prompts in portions under a token budget, then 200 decode steps replayed from graphs,
    states and windows carried all the way.  Every produced token is the plain model's choice wherever that is clear,
    and in 32-bit the logits of the last step agree."""
    folder, oracle = folders[name]
    V = CONFIGS[name]["vocab"]
    prompts = [tokens(60, 70, V), tokens(61, 3, V), tokens(62, 129, V)]
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
    assert clear >= sum(news) // 10
    if dtype == "float32":
        assert float(row_error(last["row"], ref["0"][-1]) / lim["0"][-1]) < 1.0


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
    oracle = plain.PlainZepilorn(CONFIGS["A"], read_safetensors(os.path.join(folder, "model.safetensors")))
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


_ROT_M = dict(base=1e4, dims=40, scaling=yarn(4.0, 256, 32.0, 1.0))
MID = model(1000, 320, [
    layer(attention(10, 5, 80, 48, 1.1, 130, **_ROT_M), 512),
    layer(latent(5, 48, 72, 384, 0.15, 200), 640),
    layer(linear(96, 64, [0.9, 0.99]), 256),
    layer(attention(15, 5, 80, 48, 0.9, 65, kv_from=0, **_ROT_M)),
    layer(attention(4, 4, 96, 128, 0.8, 64), 320),
    layer(linear(24, 72, [0.5, 0.95, 0.997, 1.0, 0.8]), 192)], eps=1e-6)

_ROT_O = dict(base=20.0, dims=2, scaling=yarn(3.0, 64, 2.0, 1.0))
ODD = model(1001, 200, [
    layer(latent(1, 130, 7, 600, 0.1, 64), 33),
    layer(attention(2, 2, 160, 72, 1.0, 33, base=1e4, scaling=yarn(2.0, 512, 32.0, 1.0)), 88),
    layer(attention(12, 4, 16, 8, 1.5, 65, **_ROT_O), 7),
    layer(linear(200, 300, [0.98]), 24),
    layer(attention(4, 4, 16, 8, 0.6, 2, kv_from=2, **_ROT_O), 40),
    layer(latent(33, 4, 3, 50, 0.7, 100)),
    layer(linear(4, 3, [0.1, 0.2, 0.3, 0.9, 0.99]), 88)])


@pytest.mark.parametrize("cfg,lens,tail", [(MID, [37, 130, 700], 140), (ODD, [3, 70, 260], 60)], ids=["wider", "unusual"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_other_sizes_with_a_long_request(cfg, lens, tail, dtype, tmp_path):
    """wider: sizes between the tiny configurations and a real model's (products large enough for the tensor-core
    kernels, head sizes that are no power of two, pages of 64).  unusual: heads wider than any tensor-core kernel takes
    and tiny ones, a latent of 600, a recurrent head of 200 x 300, more heads than a warp has lanes, a rotation over two
    entries, a reader that sees two tokens, a vocabulary that is no multiple of anything."""
    oracle = plain.PlainZepilorn(cfg, write_model(cfg, str(tmp_path / "m"), seed=5))
    reqs = {f"r{i}": tokens(i, n, cfg["vocab"]) for i, n in enumerate(lens)}
    ref, lim = references(oracle, reqs, dtype)
    eng = gpu_engine(str(tmp_path / "m"), dtype, page_size=64, num_pages=32)
    mixed, _ = cuttings.mixed(reqs, max_live=3, seed=2, decode_tail=40)
    for what, steps in (("whole", cuttings.whole(reqs)), ("decode", cuttings.tail_decode(reqs, tail)),
                        ("portions", cuttings.portions(reqs)), ("mixed", mixed)):
        check(cuttings.run_trace(eng, steps), ref, lim, dtype, what)
