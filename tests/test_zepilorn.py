"""Zepilorn without a GPU: the config reader and registry, tensor names and shapes, the plain implementation's own
hand-made cases (one per mechanism), and the engine's host side (cache, shared keys and values, state slots, step
function, scheduler, replay) with the plain PyTorch statement of the kernels standing in for them."""
import copy
import io
import json
import math
import os
import sys

import numpy as np
import pytest
import torch

import cuttings
import plain_zepilorn as plain
from plain_ops import PlainOps
from zepilorn_models import (CONFIGS, TOL, attention, latent, layer, linear, make_weights, one_layer, row_error, tokens,
                             write_model, yarn)

F64 = torch.float64


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("zepilorn")
    out = {}
    for name, cfg in CONFIGS.items():
        folder = str(base / name)
        out[name] = (folder, plain.PlainZepilorn(cfg, write_model(cfg, folder, seed=ord(name))))
    return out


def cpu_engine(folder, **kw):
    from dlm_b200.engine import Engine
    args = dict(dtype="float32", device="cpu", ops=PlainOps(), page_size=16, num_pages=40, max_requests=4)
    args.update(kw)
    return Engine.from_pretrained(folder, **args)


# ------------------------------------------------------------------ config, registry, tensors
def test_registry_resolves_the_architecture_and_round_trips_the_config():
    from dlm_b200.config import ZepilornConfig
    from dlm_b200.registry import architectures, resolve
    assert "Zepilorn" in architectures()
    for cfg in CONFIGS.values():
        name, typed, spec = resolve(copy.deepcopy(cfg))
        assert name == "Zepilorn" and isinstance(typed, ZepilornConfig)
        assert len(spec.layers) == len(cfg["layers"]) and spec.vocab_size == cfg["vocab"]
        assert not spec.tie_word_embeddings and spec.dependent_launch is False
        assert [c.reads_cache_of for c in spec.order] == [L["mixer"].get("kv_from") for L in cfg["layers"]]
        assert ZepilornConfig.from_dict(typed.to_dict()) == typed
        assert typed.to_dict()["layers"] == cfg["layers"]


@pytest.mark.parametrize("edit,what", [
    (lambda c: c.pop("layers"), "layers"),
    (lambda c: c.pop("width"), "width"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c["layers"][0].update(type="parallel"), "type"),
    (lambda c: c["layers"][0].pop("mixer"), "mixer"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(base=-1.0), "base"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, "x", 0.5]), "decay"),
    (lambda c: c["layers"][3]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=8), "vdim"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "mlp"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
])
def test_config_refusals(edit, what):
    from dlm_b200.config import ConfigError
    from dlm_b200.registry import resolve
    cfg = copy.deepcopy(CONFIGS["A"])
    edit(cfg)
    with pytest.raises(ConfigError) as e:
        resolve(cfg)
    assert what in str(e.value)


def test_tensor_names_and_shapes_are_the_checkpoints_own():
    from dlm_b200.parts import DecoderModel, Runtime, WeightError
    from dlm_b200.registry import resolve
    for cfg in CONFIGS.values():
        _, _, spec = resolve(copy.deepcopy(cfg))
        m = DecoderModel(spec, Runtime("cpu", torch.float32, None))
        tensors = make_weights(cfg)
        m.check({n: (t.dtype, tuple(t.shape)) for n, t in tensors.items()})
        assert set(m.param_specs()) - {"head"} == set(tensors) - {"head"}
    _, _, spec = resolve(copy.deepcopy(CONFIGS["A"]))
    m = DecoderModel(spec, Runtime("cpu", torch.float32, None))
    bad = make_weights(CONFIGS["A"])
    bad.pop("l0.norm1.b")
    bad.pop("l1.ls2")
    bad.pop("l1.mix.norm")
    bad["l2.mix.k"] = torch.zeros(72, 96)                 # a reader has no key projection
    bad["l2.norm2"] = torch.zeros(96)                     # ... and this one no feed-forward
    bad["l3.mix.dkv.norm"] = torch.zeros(27)
    with pytest.raises(WeightError) as e:
        m.check({n: (t.dtype, tuple(t.shape)) for n, t in bad.items()})
    for n in ("l0.norm1.b", "l1.ls2", "l1.mix.norm", "l2.mix.k", "l2.norm2", "l3.mix.dkv.norm"):
        assert n in str(e.value)


def test_random_weights_for_a_config_build_and_load(tmp_path):
    from dlm_b200.config import ZepilornConfig
    from dlm_b200.engine import Engine
    from dlm_b200.weights import write_random_model
    cfg = ZepilornConfig.from_dict(copy.deepcopy(CONFIGS["D"]))
    folder = write_random_model(cfg, 5, str(tmp_path / "m"))
    toks = tokens(1, 20, cfg.vocab)
    a = cpu_engine(folder)
    b = Engine.from_random(cfg, 5, dtype="float32", device="cpu", ops=PlainOps(), page_size=16, num_pages=8, max_requests=2)
    sa, sb = a.cache.open(), b.cache.open()
    la, lb = a.step([(sa, toks, [19])]), b.step([(sb, toks, [19])])
    assert torch.allclose(la, lb, atol=1e-5) and torch.isfinite(la).all() and float(la.std()) > 0


def test_blended_rotary_table():
    """The package's table against the plain statement, and the regimes by hand."""
    from dlm_b200.parts import PartSpec, Runtime
    from dlm_b200.registry import build_part
    rt = Runtime("cpu", torch.float32, None)
    for base, dims, sc in ((5000.0, 16, yarn(6.0, 96, 8.0, 0.5)), (300.0, 20, yarn(2.0, 4096, 32.0, 1.0)), (1e4, 8, None),
                           (50.0, 12, yarn(3.0, 64, 1e9, 1e-9)), (1e6, 64, yarn(1.0, 256, 16.0, 1.0)),
                           (1e4, 32, yarn(8.0, 2.0, 1.0, 0.9))):
        part = build_part("position", PartSpec("rope_yarn_neox", {"head_dim": 80, "theta": base, "rotary_dim": dims,
                                                                  "scaling": sc}))
        table, n = part.rotary(rt)
        f, amp = plain.yarn(base, dims, sc)
        assert n == dims and torch.allclose(table.double(), f, rtol=1e-7) and part.amplitude == pytest.approx(amp, abs=1e-15)
    # original 2 pi 100, fast 10, slow 1: with base 10 and dims 20, turn(10) = 10 * log10(10) = 10 and turn(1) = 20 (cut
    # to 19): pairs up to 10 would keep their frequency, and there are ten pairs, so all do
    f, amp = plain.yarn(10.0, 20, yarn(5.0, 2 * math.pi * 100, 10.0, 1.0))
    assert torch.allclose(f, torch.tensor([10.0 ** (-i / 10) for i in range(10)], dtype=F64))
    assert amp == pytest.approx(0.1 * math.log(5.0) + 1.0)
    # fast 100 / slow 10 (just below each power, so that no floor or ceiling sits on an edge): pairs 0 .. 10 blend
    f, _ = plain.yarn(10.0, 20, yarn(5.0, 2 * math.pi * 100 * 1.01, 100.0, 10.2))
    for i in range(10):
        own = 10.0 ** (-i / 10)
        assert float(f[i]) == pytest.approx(own / 5.0 * (i / 10) + own * (1 - i / 10), rel=1e-12)


# ------------------------------------------------- the plain implementation's own hand-made cases
def _mix_tensors(cfg, seed=3):
    t = {k: v.to(F64) for k, v in make_weights(cfg, seed).items()}
    return t, (lambda n: t["l0.mix." + n])


def test_plain_attention_sink_window_and_order_of_rotation_and_norm():
    """With zero queries every score is 0: n visible keys and the sink share the weight equally, so the output is
    n / (n + 1) times the mean of the visible values.  Unit heads have a root mean square of 1 (up to eps) after the
    rotation even though its amplitude stretches part of them."""
    m = attention(2, 1, 6, 3, 0.5, 4, 100.0, 4, yarn(7.0, 64, 8.0, 1.0))
    t, p = _mix_tensors(one_layer(layer(m), width=10))
    t["l0.mix.q"].zero_()
    h = torch.randn(9, 10, dtype=F64, generator=torch.Generator().manual_seed(3))
    kv = plain.attention_keys_values(h, p, m, 1e-9)
    assert torch.allclose((kv[0] ** 2).mean(-1), torch.ones(9, 1, dtype=F64), atol=1e-6)
    out = plain.windowed_attention(h, p, m, 1e-9, kv)
    for i in range(9):
        n = min(i + 1, 4)
        o = kv[1][i + 1 - n:i + 1, 0].mean(0) * n / (n + 1)
        assert torch.allclose(out[i], o.repeat(2) @ p("o").T, rtol=1e-10, atol=1e-12)
    # a large eps shows that the norm comes behind the rotation: the stretched head is what is measured
    x = torch.ones(1, 1, 6, dtype=F64)
    amp = plain.yarn(100.0, 4, m["rot"]["scaling"])[1]
    u = plain.rotated_unit_heads(x, m, 0.5)
    assert torch.allclose(u[0, 0, 4:], torch.full((2,), 1.0 / math.sqrt((4 * amp * amp + 2) / 6 + 0.5), dtype=F64))


def test_plain_attention_scores_depend_on_the_distance_only_where_rotated():
    f, amp = plain.yarn(100.0, 4, yarn(3.0, 64, 8.0, 1.0))
    g = torch.Generator().manual_seed(5)
    q, k = torch.randn(1, 1, 6, dtype=F64, generator=g), torch.randn(1, 1, 6, dtype=F64, generator=g)

    def score(i, j):
        return float((plain.rotate_halves(q, torch.tensor([i]), f, 4, amp) * plain.rotate_halves(k, torch.tensor([j]), f, 4, amp)).sum())
    assert score(9, 4) == pytest.approx(score(105, 100), rel=1e-9)
    assert score(9, 4) != pytest.approx(score(9, 5), rel=1e-3)
    assert torch.equal(plain.rotate_halves(q, torch.tensor([7]), f, 4, amp)[..., 4:], q[..., 4:])
    assert score(0, 0) == pytest.approx(float((q[..., :4] * k[..., :4]).sum() * amp ** 2 + (q[..., 4:] * k[..., 4:]).sum()))


def test_plain_latent_attention_first_token_and_window():
    """The first position sees itself only: its output is W_o W_uv c.  With a window of one every position does."""
    for window in (1, 3):
        m = latent(2, 3, 5, 7, 0.4, window)
        t, p = _mix_tensors(one_layer(layer(m), width=12))
        h = torch.randn(6, 12, dtype=F64, generator=torch.Generator().manual_seed(1))
        c = h @ p("dkv").T
        c = c / torch.sqrt((c * c).mean(-1, keepdim=True) + 1e-5) * p("dkv.norm")
        alone = (c @ p("uv").T) @ p("o").T
        out = plain.latent_attention(h, p, m, 1e-5)
        assert torch.allclose(out[0], alone[0], rtol=1e-10)
        assert torch.allclose(out, alone, rtol=1e-10) == (window == 1)


def test_plain_linear_attention_is_the_decayed_sum_over_the_past():
    m = linear(3, 5, [0.6, 0.9])
    t, p = _mix_tensors(one_layer(layer(m), width=12))
    T = 7
    h = torch.randn(T, 12, dtype=F64, generator=torch.Generator().manual_seed(2))
    got, S = plain.lightning(h, p, m, 1e-5)
    act = lambda z: z / (1 + torch.exp(-z))
    q, k = act(h @ p("q").T).reshape(T, 2, 3), act(h @ p("k").T).reshape(T, 2, 3)
    v = act(h @ p("v").T).reshape(T, 2, 5)
    o = torch.zeros(T, 2, 5, dtype=F64)
    for i in range(T):
        for j in range(i + 1):
            for n, a in enumerate((0.6, 0.9)):
                o[i, n] += a ** (i - j) * (q[i, n] @ k[j, n]) * v[j, n]
    y = o.reshape(T, 10)
    y = y / torch.sqrt((y * y).mean(-1, keepdim=True) + 1e-5) * p("norm") / (1 + torch.exp(-(h @ p("g").T)))
    assert torch.allclose(got, y @ p("o").T, rtol=1e-9)
    a, s = plain.lightning(h[:3], p, m, 1e-5)
    b, s2 = plain.lightning(h[3:], p, m, 1e-5, state=s)
    assert torch.allclose(torch.cat([a, b]), got, rtol=1e-12) and torch.allclose(s2, S)


def test_plain_layer_norm_mlp_and_order():
    x = torch.tensor([[1.0, 2.0, 3.0, 6.0]], dtype=F64)
    w, b = torch.tensor([1.0, 2.0, 1.0, 0.5], dtype=F64), torch.tensor([0.0, 1.0, -1.0, 0.0], dtype=F64)
    s = math.sqrt(3.5 + 0.25)
    assert torch.allclose(plain.layer_norm(x, w, b, 0.25), torch.tensor([[-2 / s, -2 / s + 1, -1.0, 1.5 / s]], dtype=F64))
    cfg = CONFIGS["A"]
    t = make_weights(cfg, 9)
    mdl = plain.PlainZepilorn(cfg, t)
    logits, after = mdl.forward(tokens(2, 7, cfg["vocab"]), trace=True)
    t = {k: v.to(F64) for k, v in t.items()}
    # layer 1 by hand, from the residual after layer 0: both sublayers read the residual itself
    mix, _ = plain.lightning(after[0], lambda n: t["l1.mix." + n], cfg["layers"][1]["mixer"], 1e-5)
    x1 = after[0] + plain.layer_norm(mix, t["l1.norm1"], t["l1.norm1.b"], 1e-5) * t["l1.ls1"]
    gu = torch.nn.functional.gelu(x1 @ t["l1.mlp.gate"].T, approximate="tanh") * (x1 @ t["l1.mlp.up"].T)
    x2 = x1 + plain.layer_norm(gu @ t["l1.mlp.down"].T, t["l1.norm2"], t["l1.norm2.b"], 1e-5) * t["l1.ls2"]
    assert torch.allclose(after[1], x2, rtol=1e-12)
    assert torch.allclose(logits, plain.layer_norm(after[-1], t["final.norm"], t["final.norm.b"], 1e-5) @ t["head"].T)


def test_plain_reader_uses_the_earlier_layers_keys_and_values():
    """A reader's output changes with the earlier layer's key and value projections although its own input is kept."""
    cfg = CONFIGS["A"]
    mdl = plain.PlainZepilorn(cfg, make_weights(cfg, 4))
    x = torch.randn(30, 96, dtype=F64, generator=torch.Generator().manual_seed(8))
    kept = {}
    mdl.mixer(0, x, kept)
    a = mdl.mixer(2, x, kept)
    b = mdl.mixer(2, x, {0: (kept[0][0], kept[0][1] * 2.0)})
    assert torch.allclose(b, 2.0 * a) and not torch.allclose(a, torch.zeros_like(a))


# ----------------------------------------------------------------- engine host side on the CPU
@pytest.mark.parametrize("name", ["A", "B", "D"])
def test_every_cutting_matches_the_plain_model(name, folders):
    folder, oracle = folders[name]
    V = CONFIGS[name]["vocab"]
    reqs = {f"r{i}": tokens(i, n, V) for i, n in enumerate([1, 17, 41, 80])}
    ref = {rid: oracle.forward(t) for rid, t in reqs.items()}
    eng = cpu_engine(folder)
    mixed, _ = cuttings.mixed(reqs, max_live=3, seed=1)
    worst = 0.0
    for steps in (cuttings.whole(reqs), cuttings.tail_decode(reqs, 20), cuttings.portions(reqs), mixed):
        got = cuttings.run_trace(eng, steps)
        assert len(got) == sum(len(t) for t in reqs.values())
        worst = max([worst] + [float(row_error(row, ref[rid][p])) for (rid, p), row in got.items()])
    print(f"{name}: worst relative error {worst:.2e}")
    assert worst < TOL["float32"]
    assert all(p.used_pages == 0 for p in eng.cache.stats())


def test_residual_after_every_layer(folders):
    folder, oracle = folders["A"]
    toks = tokens(3, 23, CONFIGS["A"]["vocab"])
    _, after = oracle.forward(toks, trace=True)
    eng = cpu_engine(folder)
    seen = []
    eng.model.after_layer = lambda call, x: seen.append(x.detach().to(F64).clone())
    slot = eng.cache.open()
    eng.step([(slot, toks, [])])
    eng.cache.close(slot)
    assert len(seen) == after.shape[0]
    for i, x in enumerate(seen):
        assert float((x - after[i]).abs().max() / after[i].abs().max()) < 2e-5, i


def test_a_cache_keeps_what_its_furthest_reader_needs(folders):
    """Readers own no pages; the layer they read keeps as many tokens as the furthest-looking of them (all of them
    when one has no window)."""
    eng = cpu_engine(folders["A"][0])
    owners = [ci for ci in range(5) if ci in eng.cache.tensors]
    assert owners == [0, 3]
    assert sorted(eng.cache.group_windows) == [33, 45]            # layer 0: 19 of its own, readers of 45 and 7
    assert eng.cache.call_group[0] == eng.cache.call_group[2] == eng.cache.call_group[4] != eng.cache.call_group[3]
    eng = cpu_engine(folders["D"][0])
    assert eng.cache.group_windows == [0] and sorted(eng.cache.tensors) == [0, 4]
    # pages of the widened window go back to the pool as it passes
    eng = cpu_engine(folders["A"][0])
    slot = eng.cache.open()
    for i in range(0, 160, 8):
        eng.step([(slot, tokens(5, 8, 131), [])])
    used = {w: s.used_pages for w, s in zip(eng.cache.group_windows, eng.cache.stats())}
    assert used[45] <= 5 and used[33] <= 4
    eng.cache.close(slot)


def test_slots_and_pages_are_used_again_with_fresh_state(folders):
    """Six requests through three slots and a pool that holds only what is live."""
    folder, oracle = folders["A"]
    V = CONFIGS["A"]["vocab"]
    reqs = {f"q{i}": tokens(20 + i, n, V) for i, n in enumerate([70, 33, 129, 16, 90, 7])}
    steps, _ = cuttings.mixed(reqs, max_live=3, seed=2)
    eng = cpu_engine(folder, num_pages=cuttings.peak_tokens(steps) // 16, max_requests=3)
    got = cuttings.run_trace(eng, steps)
    ref = {rid: oracle.forward(t) for rid, t in reqs.items()}
    assert max(float(row_error(row, ref[rid][p])) for (rid, p), row in got.items()) < TOL["float32"]
    assert all(s.used_pages == 0 for s in eng.cache.stats())


def test_greedy_generation_through_the_scheduler(folders):
    """Engine.generate (scheduler, portions under a token budget, sampling, commit) against greedy decoding with the
    plain model; batched prompts give what each gives alone."""
    folder, oracle = folders["B"]
    V = CONFIGS["B"]["vocab"]
    prompts = [tokens(40, 5, V), tokens(41, 37, V), tokens(42, 1, V)]
    outs = cpu_engine(folder, max_step_tokens=16).generate(prompts, max_new_tokens=8)
    for p, out in zip(prompts, outs):
        seq = list(p)
        for tok in out:
            row = oracle.forward(seq)[-1]
            top2 = torch.topk(row, 2).values
            if float(top2[0] - top2[1]) > 1e-3:
                assert int(torch.argmax(row)) == tok
            seq.append(tok)
    assert [cpu_engine(folder).generate(p, max_new_tokens=8) for p in prompts] == outs


def test_replay_program_on_the_stand_in(folders, tmp_path, monkeypatch):
    from dlm_b200.engine import Engine, replay
    folder, oracle = folders["A"]
    V = CONFIGS["A"]["vocab"]
    reqs = {"a": tokens(50, 45, V), "b": tokens(51, 9, V)}
    steps, _ = cuttings.mixed(reqs, max_live=2, seed=3)
    real = Engine.from_pretrained
    monkeypatch.setattr(Engine, "from_pretrained", classmethod(
        lambda cls, path, **kw: real(path, **dict(kw, device="cpu", ops=PlainOps()))))
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"))
    out_dir = str(tmp_path / "out")
    assert replay.main(["--model", folder, "--dtype", "float32", "--out", out_dir, "--max-tokens", "128",
                        "--page-size", "16", "--device", "cpu"]) == 0
    fed = {r: 0 for r in reqs}
    for st in steps:
        rows = np.fromfile(os.path.join(out_dir, f"{st['step']}.f32"), dtype="<f4").reshape(-1, V)
        k = 0
        for e in st["entries"]:
            ref = oracle.forward(reqs[e["id"]][:fed[e["id"]] + len(e["tokens"])])
            for w in e["want"]:
                assert float(row_error(torch.from_numpy(rows[k].copy()), ref[fed[e["id"]] + w])) < TOL["float32"]
                k += 1
            fed[e["id"]] += len(e["tokens"])


@pytest.mark.parametrize("mixer", [attention(4, 2, 8, 12, 1.0, 6, 200.0, 4, yarn(4.0, 32, 4.0, 0.5)), latent(3, 8, 10, 24, 0.5, 9),
                                   linear(6, 10, [0.4, 0.99])])
@pytest.mark.parametrize("ff", [None, 20])
def test_a_single_layer_of_every_kind(mixer, ff, tmp_path):
    cfg = one_layer(layer(mixer, ff), width=32, vocab=41)
    folder = str(tmp_path / "m")
    oracle = plain.PlainZepilorn(cfg, write_model(cfg, folder, seed=5))
    reqs = {"a": tokens(1, 40, 41), "b": tokens(2, 7, 41)}
    ref = {rid: oracle.forward(t) for rid, t in reqs.items()}
    eng = cpu_engine(folder)
    mixed, _ = cuttings.mixed(reqs, max_live=2, seed=6)
    for steps in (cuttings.whole(reqs), cuttings.portions(reqs, sizes=(2, 5)), mixed):
        got = cuttings.run_trace(eng, steps)
        assert max(float(row_error(row, ref[rid][p])) for (rid, p), row in got.items()) < TOL["float32"]


def test_norm_on_outputs_with_other_norms_and_blocks():
    """The output-norm block with an RMS norm, and with a norm no kernel can apply itself, equals its plain statement;
    after a block of another kind the rounded residual is made anew."""
    from types import SimpleNamespace
    from dlm_b200.parts import PartSpec, Runtime
    from dlm_b200.parts.base import StepContext
    from dlm_b200.registry import build_part
    rt = Runtime("cpu", torch.bfloat16, PlainOps())
    W = 24
    g = torch.Generator().manual_seed(1)
    for norm in (PartSpec("rmsnorm", {"size": W, "eps": 1e-5, "param": ""}), PartSpec("dynamic_tanh", {"size": W, "param": ""}),
                 PartSpec("layernorm", {"size": W, "eps": 1e-5, "param": ""})):
        block = build_part("block", PartSpec("postnorm", {
            "norm1": norm, "mixer": PartSpec("retention", {"hidden_size": W, "heads": 2, "dim": 4, "vdim": 6,
                                                           "decay": [0.5, 0.9], "eps": 1e-5}),
            "names": {"norm1": "n1", "mixer": "m."}}))
        t = {s.name: torch.randn(*s.shape, generator=g) * 0.5 if s.shape else torch.tensor(0.7) for s in block.param_specs()}
        block.load(t, rt)
        state = torch.zeros(2, 2, 4, 6)
        batch = SimpleNamespace(num_requests=1, cu_q=torch.tensor([0, 5], dtype=torch.int32),
                                state_slot=torch.tensor([0], dtype=torch.int32), positions=torch.arange(5, dtype=torch.int32))
        ctx = StepContext(rt, batch, lambda c: None, lambda c, n="": state)
        x = torch.randn(5, W, generator=g)
        x0 = x.clone()
        block.forward(x, ctx, 0)
        y = torch.zeros(5, W)
        state.zero_()
        block.mixer.forward(x0.to(torch.bfloat16), y, ctx, 0)
        want = x0 + block.norm1.forward(y, rt, out_dtype=torch.float32)
        assert torch.allclose(x, want, atol=1e-5)
        assert torch.equal(ctx.rounded(1, x), x.to(torch.bfloat16))
        x += 1.0                                                  # call 1 was a block that leaves no copy
        assert torch.equal(ctx.rounded(2, x), x.to(torch.bfloat16))
        assert float(ctx.take_zeroed(x).abs().max()) == 0.0
    with pytest.raises(NotImplementedError):
        build_part("norm", PartSpec("dynamic_tanh", {"size": W})).scale_output(torch.ones(W))


def test_the_benchmarks_configurations_resolve():
    """The benchmark's model of this design and the one beside it: equal width, layers, feed-forward and attention
    heads; the reader's layer owns no cache."""
    import sys as _sys
    _sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    import bench
    from dlm_b200.registry import resolve
    z = bench.zepilorn_config(1024)
    _, cfg, spec = resolve(copy.deepcopy(z))
    _, q, qspec = resolve(bench.qwen_config_like_zepilorn(z))
    assert len(spec.layers) == len(qspec.layers) == 5 and spec.hidden_size == qspec.hidden_size == 1024
    att = cfg.layers[0]["mixer"]
    assert (q.num_attention_heads, q.num_key_value_heads, q.head_dim) == (att["heads"], att["kv_heads"], att["dim"])
    assert spec.order[3].reads_cache_of == 0
