"""Gakenex without a GPU: the config reader and registry, tensor names and shapes, the plain implementation's own
hand-made cases (one per mechanism), the cache manager's kept first tokens, and the engine's host side (cache, state
slots, step function, scheduler, replay) with the plain PyTorch statement of the kernels standing in for them."""
import copy
import io
import json
import math
import os
import random
import sys

import numpy as np
import pytest
import torch

import cuttings
import plain_gakenex as plain
from gakenex_models import (CONFIGS, TOL, attention, clear_requests, dense, layer, make_weights, moe, one_layer, row_error,
                            tokens, write_model)
from plain_ops import PlainOps

F64 = torch.float64


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("gakenex")
    out = {}
    for name, cfg in CONFIGS.items():
        folder = str(base / name)
        out[name] = (folder, plain.PlainGakenex(cfg, write_model(cfg, folder, seed=ord(name))))
    return out


def cpu_engine(folder, **kw):
    from dlm_b200.engine import Engine
    args = dict(dtype="float32", device="cpu", ops=PlainOps(), page_size=16, num_pages=40, max_requests=4)
    args.update(kw)
    return Engine.from_pretrained(folder, **args)


# ------------------------------------------------------------------ config, registry, tensors
def test_registry_resolves_the_architecture_and_round_trips_the_config():
    from dlm_b200.config import GakenexConfig
    from dlm_b200.registry import architectures, resolve
    assert "Gakenex" in architectures()
    for cfg in CONFIGS.values():
        name, typed, spec = resolve(copy.deepcopy(cfg))
        assert name == "Gakenex" and isinstance(typed, GakenexConfig)
        assert len(spec.layers) == len(cfg["layers"]) and spec.vocab_size == cfg["vocab"]
        assert spec.lm_head_name is None and spec.dependent_launch is False
        assert spec.logit_softcap == (cfg.get("logit_softcap") or 0.0)
        assert GakenexConfig.from_dict(typed.to_dict()) == typed
        assert typed.to_dict() == cfg


@pytest.mark.parametrize("edit,what", [
    (lambda c: c.pop("layers"), "layers"),
    (lambda c: c.pop("width"), "width"),
    (lambda c: c.pop("max_positions"), "max_positions"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(logit_softcap=-1.0), "logit_softcap"),
    (lambda c: c["layers"][0].update(type="lightning"), "type"),
    (lambda c: c["layers"][0].pop("mixer"), "mixer"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][0]["mixer"].update(dim=130), "dim"),
    (lambda c: c["layers"][0]["mixer"].update(conv=17), "conv"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "mlp"),
    (lambda c: c["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=10), "router.top"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), "expert"),
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
        assert set(m.param_specs()) == set(tensors)
    _, _, spec = resolve(copy.deepcopy(CONFIGS["A"]))
    m = DecoderModel(spec, Runtime("cpu", torch.float32, None))
    bad = make_weights(CONFIGS["A"])
    for n in ("pos", "embed.norm", "l0.mix.q.conv", "l1.mix.lk2", "l1.mlp.e8.up"):
        bad.pop(n)
    bad["l2.norm2"] = torch.zeros(96)                     # a layer has one norm
    bad["l1.mlp.router"] = torch.zeros(8, 96)
    with pytest.raises(WeightError) as e:
        m.check({n: (t.dtype, tuple(t.shape)) for n, t in bad.items()})
    for n in ("pos", "embed.norm", "l0.mix.q.conv", "l1.mix.lk2", "l1.mlp.e8.up", "l2.norm2", "l1.mlp.router"):
        assert n in str(e.value)


def test_random_weights_for_a_config_build_and_load(tmp_path):
    from dlm_b200.config import GakenexConfig
    from dlm_b200.engine import Engine
    from dlm_b200.weights import write_random_model
    cfg = GakenexConfig.from_dict(copy.deepcopy(CONFIGS["D"]))
    folder = write_random_model(cfg, 5, str(tmp_path / "m"))
    toks = tokens(1, 20, cfg.vocab)
    a = cpu_engine(folder)
    b = Engine.from_random(cfg, 5, dtype="float32", device="cpu", ops=PlainOps(), page_size=16, num_pages=8, max_requests=2)
    sa, sb = a.cache.open(), b.cache.open()
    la, lb = a.step([(sa, toks, [19])]), b.step([(sb, toks, [19])])
    assert torch.allclose(la, lb, atol=1e-5) and torch.isfinite(la).all() and float(la.std()) > 0
    # weights stored around zero: the norms a random model gets are close to one
    assert float((a.model.final_norm.weight - 1.0).abs().max()) < 0.2


# ------------------------------------------------- the plain implementation's own hand-made cases
def _mix_tensors(cfg, seed=3):
    t = {k: v.to(F64) for k, v in make_weights(cfg, seed).items()}
    return t, (lambda n: t["l0.mix." + n])


def rnd(*shape, seed=1):
    return torch.randn(*shape, dtype=F64, generator=torch.Generator().manual_seed(seed))


def test_plain_short_convolution():
    u = torch.tensor([[1.0], [10.0], [100.0], [1000.0]], dtype=F64)
    w = torch.tensor([[2.0, 3.0, 5.0]], dtype=F64)            # the last tap meets the current token
    assert plain.short_conv(u, w).flatten().tolist() == [5.0, 53.0, 532.0, 5320.0]


def test_plain_visibility():
    see = plain.visible(8, {"size": 2, "keep_first": 3})
    assert see[7].tolist() == [True, True, True, False, False, False, True, True]
    assert see[1].tolist() == [True, True] + [False] * 6            # a kept token is not seen before it is there
    assert see[3].tolist() == [True, True, True, True] + [False] * 4
    assert plain.visible(5, {"size": 1})[4].tolist() == [False] * 4 + [True]
    assert bool(plain.visible(5, None)[4].all())


def test_plain_attention_with_zero_queries_is_the_difference_of_equal_means():
    """Zero queries: both maps give the mean of the visible values, so a head is (1 - lambda) mean, divided by its root
    mean square: its size is gone and its sign is that of 1 - lambda."""
    for shift, sign in ((0.0, 1.0), (1.0, -1.0)):
        m = attention(2, 1, 6, 5, 0.5, 0.3, None, 3, 2)
        t, p = _mix_tensors(one_layer(layer(m), width=10))
        t["l0.mix.q"].zero_()
        t["l0.mix.g"].zero_()                                         # a gate of one half
        t["l0.mix.lk1"] += shift
        assert (1.0 - plain.mixing_factor(p, 0.3) > 0) == (sign > 0)
        h = rnd(9, 10)
        v = h @ p("v").T
        out = plain.differential_attention(h, p, m, 1e-12)
        for i in range(9):
            js = sorted(set(range(max(0, i - 2), i + 1)) | set(range(min(2, i + 1))))
            mean = v[js].mean(0)
            o = sign * mean / torch.sqrt((mean * mean).mean()) * 0.7 * 0.5
            assert torch.allclose(out[i], o.repeat(2) @ p("o").T, rtol=1e-6), i


def test_plain_attention_layout_of_maps_and_groups():
    """Loud equal entries of one map's query and of its key's map meet; the other map stays flat.  Query heads share
    keys and values group by group."""
    m = attention(4, 2, 3, 2, 1.0, 0.2, None)
    t, p = _mix_tensors(one_layer(layer(m), width=16))
    h = torch.eye(16, dtype=F64)[:6]
    q, k = t["l0.mix.q"], t["l0.mix.k"]
    q.zero_(), k.zero_()
    t["l0.mix.q.norm"].fill_(1.0), t["l0.mix.k.norm"].fill_(6.0)
    q.view(4, 2, 3, 16)[:, :, 0, 5] = 1.0                              # token 5 asks in every head and map
    k.view(2, 2, 3, 16)[:, :, 1, :6] = 1.0                             # every key is orthogonal to it ...
    k.view(2, 2, 3, 16)[1, 1, :, 2] = torch.tensor([1.0, 0.0, 0.0])    # ... but token 2's in group 1, map 2
    a = plain.differential_maps(h, p, m, 1e-12)
    v = (h @ p("v").T).reshape(6, 2, 2)
    flat = v.mean(0)
    for n in range(4):
        for c in range(2):
            want = v[2, 1] if (n // 2, c) == (1, 1) else flat[n // 2]
            assert torch.allclose(a[5, n, c], want, rtol=1e-3, atol=1e-3), (n, c)


def test_plain_mixing_factor():
    t = {"lq1": [1.0, 2.0], "lk1": [0.5, 0.25], "lq2": [3.0, 0.0], "lk2": [-0.5, 9.0]}
    assert plain.mixing_factor(lambda n: torch.tensor(t[n], dtype=F64), 0.4) == \
        pytest.approx(math.exp(1.0) - math.exp(-1.5) + 0.4)


def test_plain_clamped_mlp():
    eye = {"gate": torch.eye(4, dtype=F64), "up": torch.diag(torch.tensor([1.0, -9.0, 9.0, 0.25], dtype=F64)), "down": torch.eye(4, dtype=F64)}
    y = plain.clamped_mlp(torch.tensor([[5.0, 1.0, -3.0, -40.0]], dtype=F64), lambda n: eye[n], 2.0)[0]
    s = lambda z: 1.0 / (1.0 + math.exp(-1.702 * z))
    # gate 5 -> 2, up 5 -> 2; gate 1, up -9 -> -2; gate -3 (no lower limit), up -27 -> -2; gate -40, up -10 -> -2
    want = [2 * s(2) * 3, s(1) * -1, -3 * s(-3) * -1, -40 * s(-40) * -1]
    assert torch.allclose(y, torch.tensor(want, dtype=F64))


def test_plain_experts_weigh_their_input():
    """A weight of one half in front of an expert is not one half behind it; weights are the scores themselves."""
    cfg = one_layer(layer(attention(1, 1, 2, 2, 1.0, 0.1), moe(4, 2, 6)), width=8)
    t = {k: v.to(F64) for k, v in make_weights(cfg, 4).items()}
    p = lambda n: t["l0.mlp." + n]
    h = rnd(5, 8)
    z = h @ p("router").T
    s = 1.0 / (1.0 + torch.exp(-z))
    out = plain.weighted_input_experts(h, p, 2)
    for i in range(5):
        want = torch.zeros(8, dtype=F64)
        for e in torch.topk(z[i], 2).indices.tolist():
            x = s[i, e] * h[i]
            g, u = p(f"e{e}.gate") @ x, p(f"e{e}.up") @ x
            want += p(f"e{e}.down") @ (g / (1 + torch.exp(-g)) * u)
        assert torch.allclose(out[i], want, rtol=1e-10)
        behind = sum(float(s[i, e]) * plain.expert(h[i:i + 1], p, e)[0] for e in torch.topk(z[i], 2).indices.tolist())
        assert not torch.allclose(out[i], behind, rtol=1e-2)


def test_plain_norms_layers_and_head():
    x = torch.tensor([[3.0, 4.0]], dtype=F64)
    w = torch.tensor([0.5, -1.0], dtype=F64)
    assert torch.allclose(plain.model_norm(x, w, 0.5), torch.tensor([[3.0 * 1.5 / math.sqrt(13.0), 0.0]], dtype=F64))
    cfg = CONFIGS["A"]
    mdl = plain.PlainGakenex(cfg, make_weights(cfg, 9))
    t, toks = mdl.t, tokens(2, 7, 131)
    logits, after = mdl.forward(toks, trace=True)
    e = t["embed"][toks] + t["pos"][:7]
    x0 = e / torch.sqrt((e * e).mean(-1, keepdim=True) + 1e-5) * (1 + t["embed.norm"])
    h = x0 / torch.sqrt((x0 * x0).mean(-1, keepdim=True) + 1e-5) * (1 + t["l0.norm1"])
    # both sublayers read the same normed rows
    mix = plain.differential_attention(h, lambda n: t["l0.mix." + n], cfg["layers"][0]["mixer"], 1e-5)
    ff = plain.clamped_mlp(h, lambda n: t["l0.mlp." + n], 1.5)
    assert torch.allclose(after[0], x0 + mix + ff, rtol=1e-12)
    z = plain.model_norm(after[-1], t["final.norm"], 1e-5) @ t["embed"].T
    assert torch.allclose(logits, 12.0 * torch.tanh(z / 12.0)) and float(z.abs().max()) > 12.0


# ------------------------------------------------------------ the cache manager's kept first tokens
def manager(pages, page, window, keep, slots=4):
    from dlm_b200.build import load_host
    host = load_host()
    return host.CacheManager([host.GroupSpec(page, window, pages, keep)], slots)


def test_kept_pages_stay_while_the_window_passes():
    m = manager(12, 16, 20, 33)                       # the first 33 positions lie in pages 0, 1 and 2
    s = m.open()
    for _ in range(40):
        m.append([(s, 4)])
    t = m.table(s, 0)
    assert len(t) == 10 and all(p >= 0 for p in t[:3]) and t[3:7] == [-1] * 4 and all(p >= 0 for p in t[8:])
    # the next query is at 160 and sees back to 141 (page 8); page 7 went when position 160 was not yet there
    m.append([(s, 1)])
    assert m.table(s, 0)[7] == -1 and m.stats(0).used_pages == 3 + 3
    assert m.check() == ""
    m.close(s)
    assert m.stats(0).used_pages == 0
    # nothing is given back while everything is kept, and kept pages are handed on after the end
    m = manager(4, 16, 1, 64)
    s = m.open()
    m.append([(s, 60)])
    m.append([(s, 4)])
    assert m.stats(0).used_pages == 4 and m.pages_needed(s, 0) == [0]
    m.close(s)
    s = m.open()
    m.append([(s, 64)])
    assert m.check() == ""


def test_kept_tokens_must_not_be_negative():
    with pytest.raises(ValueError):
        manager(4, 16, 8, -1)


@pytest.mark.parametrize("seed", [0, 1, 2])
def test_random_traffic_with_kept_tokens(seed):
    """Whatever the order, every page of a kept or a visible position is there, and no page is lost or held twice."""
    rng = random.Random(seed)
    page, window, keep = rng.choice([(16, 20, 33), (8, 3, 9), (16, 50, 5)])
    m = manager(40, page, window, keep)
    live = {}
    for _ in range(400):
        if len(live) < 4 and rng.random() < 0.2:
            live[m.open()] = 0
        for s in list(live):
            n = rng.choice([1, 1, 1, 2, 7, 30])
            if rng.random() < 0.05 or not m.can_append([(s, n)]):
                m.close(s)
                del live[s]
                continue
            m.append([(s, n)])
            live[s] += n
            t = m.table(s, 0)
            for first in (live[s] - n,):
                seen = set(range(min(keep, live[s]))) | set(range(max(0, first - window + 1), live[s]))
            assert all(t[j // page] >= 0 for j in seen)
        assert m.check() == ""


# ----------------------------------------------------------------- engine host side on the CPU
@pytest.mark.parametrize("name", ["A", "B", "D"])
def test_every_cutting_matches_the_plain_model(name, folders):
    folder, oracle = folders[name]
    reqs = clear_requests(oracle, [1, 17, 41, 80])
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


def test_groups_and_pages_of_a_long_request(folders):
    """Layers with the same window and kept tokens share a pool; a long request holds its kept pages and its window's."""
    eng = cpu_engine(folders["A"][0])
    assert list(zip(eng.cache.group_windows, eng.cache.group_keep)) == [(19, 21), (37, 5), (50, 33)]
    assert eng.cache.call_group[0] == eng.cache.call_group[2]
    slot = eng.cache.open()
    for i in range(0, 240, 8):
        eng.step([(slot, tokens(5 + i, 8, 131), [])])
    used = {w: s.used_pages for w, s in zip(eng.cache.group_windows, eng.cache.stats())}
    assert used[19] <= 2 + 3 and used[37] <= 1 + 4 and used[50] <= 3 + 5
    eng.cache.close(slot)
    eng = cpu_engine(folders["D"][0])
    assert list(zip(eng.cache.group_windows, eng.cache.group_keep)) == [(0, 0), (11, 0), (6, 40)]


def test_slots_and_pages_are_used_again_with_fresh_state(folders):
    """Six requests through three slots and a pool that holds only what is live."""
    folder, oracle = folders["A"]
    reqs = clear_requests(oracle, [70, 33, 129, 16, 90, 7], seed=3)
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


@pytest.mark.parametrize("mlp", [None, dense(20, 0.8), moe(4, 2, 18)])
@pytest.mark.parametrize("mixer", [attention(4, 2, 8, 12, 0.8, 0.3, 3, 6, 9), attention(3, 1, 6, 20, 0.6, 0.7)])
def test_a_single_layer_of_every_kind(mixer, mlp, tmp_path):
    cfg = one_layer(layer(mixer, mlp), width=32, vocab=41)
    folder = str(tmp_path / "m")
    oracle = plain.PlainGakenex(cfg, write_model(cfg, folder, seed=5))
    reqs = clear_requests(oracle, [40, 7])
    ref = {rid: oracle.forward(t) for rid, t in reqs.items()}
    eng = cpu_engine(folder)
    mixed, _ = cuttings.mixed(reqs, max_live=2, seed=6)
    for steps in (cuttings.whole(reqs), cuttings.portions(reqs, sizes=(2, 5)), mixed):
        got = cuttings.run_trace(eng, steps)
        assert max(float(row_error(row, ref[rid][p])) for (rid, p), row in got.items()) < TOL["float32"]


def test_parts_serve_other_designs():
    """The new parts take their constants as parameters: a kept start beside a window in the other attention mixer, an
    RMS norm with any offset, experts weighted at their input with softmax scores, a parallel block with one norm or two."""
    from dlm_b200.parts import PartSpec, Runtime
    from dlm_b200.registry import build_part
    rt = Runtime("cpu", torch.float32, PlainOps())
    a = build_part("mixer", PartSpec("head_normed_attention", {
        "hidden_size": 16, "heads": 2, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 1.0, "eps": 1e-5, "window": 9, "keep_first": 4}))
    assert (a.cache_need().window, a.cache_need().keep_first) == (9, 4)
    with pytest.raises(ValueError):
        build_part("mixer", PartSpec("head_normed_attention", {
            "hidden_size": 16, "heads": 2, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 1.0, "eps": 1e-5, "window": 9,
            "chunk": 8, "keep_first": 4}))
    with pytest.raises(ValueError):
        build_part("mixer", PartSpec("differential_attention", {
            "hidden_size": 16, "heads": 2, "kv_heads": 1, "dim": 129, "vdim": 8, "scale": 1.0, "eps": 1e-5, "diff": 0.1}))
    n = build_part("norm", PartSpec("rmsnorm", {"size": 4, "eps": 1e-5, "offset": 0.5}))
    n.load({"weight": torch.tensor([0.0, 1.0, -0.5, 2.0])}, rt)
    assert n.weight.tolist() == [0.5, 1.5, 0.0, 2.5]
    g = torch.Generator().manual_seed(1)
    f = build_part("ffn", PartSpec("moe_topk", {"hidden_size": 8, "num_experts": 3, "top_k": 2, "expert_intermediate_size": 6,
                                                "norm_topk_prob": True, "score": "softmax", "weigh": "input"}))
    t = {s.name: torch.randn(*s.shape, generator=g) for s in f.param_specs()}
    f.load(t, rt)
    h, resid = torch.randn(5, 8, generator=g), torch.zeros(5, 8)
    ctx = type("Ctx", (), {"rt": rt})()
    f.forward(h, resid, ctx)
    prob = torch.softmax(h @ t["gate.weight"].T, dim=-1)
    for i in range(5):
        top = torch.topk(prob[i], 2)
        want = torch.zeros(8)
        for w, e in zip(top.values / top.values.sum(), top.indices.tolist()):
            x = w * h[i]
            want += t[f"experts.{e}.down_proj.weight"] @ (torch.nn.functional.silu(t[f"experts.{e}.gate_proj.weight"] @ x)
                                                          * (t[f"experts.{e}.up_proj.weight"] @ x))
        assert torch.allclose(resid[i], want, atol=1e-4, rtol=1e-4)
    with pytest.raises(ValueError):
        build_part("ffn", PartSpec("moe_topk", {"hidden_size": 8, "num_experts": 3, "top_k": 2, "expert_intermediate_size": 6,
                                                "norm_topk_prob": True, "score": "tanh"}))


def test_a_reader_widens_window_and_kept_start():
    """A cache that other calls read keeps the longest window and the most first tokens among them."""
    from dlm_b200.parts import DecoderModel, LayerCall, ModelSpec, PartSpec, Runtime
    att = lambda w, k, own: PartSpec("parallel", {"norm1": PartSpec("rmsnorm", {"size": 16, "eps": 1e-5}), "mixer": PartSpec(
        "head_normed_attention", {"hidden_size": 16, "heads": 2, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 1.0, "eps": 1e-5,
                                  "window": w, "keep_first": k, "own_kv": own})})
    spec = ModelSpec(hidden_size=16, vocab_size=20, layers=[att(9, 4, True), att(5, 7, False)], layer_prefixes=["a.", "b."],
                     final_norm=PartSpec("rmsnorm", {"size": 16, "eps": 1e-5}), order=[LayerCall(0), LayerCall(1, reads_cache_of=0)])
    need = DecoderModel(spec, Runtime("cpu", torch.float32, None)).cache_needs()[0][0]
    assert (need.window, need.keep_first) == (9, 7)


def test_the_benchmarks_configurations_resolve():
    """The benchmark's model of this design and the one beside it: equal width, layers, feed-forwards, heads and window."""
    sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    import bench
    from dlm_b200.registry import resolve
    z = bench.gakenex_config(1024)
    _, cfg, spec = resolve(copy.deepcopy(z))
    _, q, qspec = resolve(bench.qwen_config_like_gakenex(z))
    assert len(spec.layers) == len(qspec.layers) == 4 and spec.hidden_size == qspec.hidden_size == 1024
    att = cfg.layers[0]["mixer"]
    assert (q.num_attention_heads, q.num_key_value_heads, q.head_dim) == (att["heads"], att["kv_heads"], att["vdim"])
    assert [L.params["ffn"].kind for L in spec.layers] == ["clamped_glu_dense", "moe_topk"] * 2
    assert [L.params["ffn"].kind for L in qspec.layers] == ["swiglu_dense", "moe_softmax_topk"] * 2
