"""Fovosun without a GPU: configuration and weights, the plain implementation's own mechanisms on hand-made inputs, and the
engine's host logic (pages of windows, state slots of memories and convolution tails, portions, mixed batches) with the
kernels replaced by the CPU stand-in, against the plain implementation."""
import json
import math

import pytest
import torch

import fovosun_cases as fo
import helpers
import plain_fovosun as pl
from kungfu_b200 import api, registry
from kungfu_b200.config.base import ConfigError
from kungfu_b200.weights.store import WeightError, WeightStore

D64 = torch.float64


def _runner(folder, page, max_tokens, max_requests=4):
    cfg, model = api.load_model(folder, dtype="float32", device="cpu")
    return api.make_runner(cfg, model, dtype="float32", device="cpu", page_size=page, max_tokens=max_tokens,
                           max_requests=max_requests, max_context=512)


def _rel(got, ref):
    assert got
    scale = max(float(r.abs().max()) for r in ref.values())
    return max(float((row - ref[rid][pos].float()).abs().max()) for (rid, pos), row in got.items()) / scale


def test_config_reads_every_size_and_round_trips():
    cfg = api.load_config(json.loads(json.dumps(fo.FO_A)))
    assert (cfg.architecture, cfg.width, cfg.vocab, cfg.streams, len(cfg.layers)) == ("Fovosun", 64, 300, 2, 3)
    assert (cfg.norm_eps, cfg.embedding_scale) == (1e-6, 1.7)
    b, r, a = (x.mixer for x in cfg.layers)
    assert (b.heads, b.kv_heads, b.dim, b.vdim, b.scale, b.diff, b.window, b.rot_base, b.rot_dims) == (4, 2, 12, 16, 0.4, 0.3, 9, 100.0, 8)
    assert b.taps == 0 and b.temperature is None
    assert (r.heads, r.dim, r.vdim, r.decay, r.rot_base, r.rot_dims) == (3, 16, 8, (0.5, 0.9, 0.995), 50.0, 16)
    assert (a.taps, a.temperature, a.window, a.rot_dims) == (4, (0.7, 5), None, 0)
    f = cfg.layers[0].mlp
    assert (f.kind, f.ffn.ff, f.ffn.limit, f.experts, f.top, f.shared.ff, f.shared.limit) == ("moe", 24, 1.3, 5, 2, 40, 0.6)
    assert cfg.layers[1].mlp is None and (cfg.layers[2].mlp.kind, cfg.layers[2].mlp.ffn.limit) == ("dense", 0.9)
    for case in (fo.FO_A, fo.FO_B, fo.FO_C, fo.FO_D, fo.FO_E):
        c = api.load_config(json.loads(json.dumps(case)))
        assert api.load_config(json.loads(json.dumps(c.to_dict()))) == c
    rows = cfg.state_summary()
    assert rows[0]["window"] == 9 and rows[0]["bytes_per_token"] == 2 * 2 * 32 * 2 and rows[0]["fixed_bytes"] == 0
    assert rows[1]["fixed_bytes"] == 4 * 3 * 16 * 8 and rows[1]["bytes_per_token"] == 0
    assert rows[2]["fixed_bytes"] == 4 * 3 * (2 * 9 * 8 + 3 * 20)


@pytest.mark.parametrize("change,word", [
    (lambda c: c.pop("streams"), "streams"),
    (lambda c: c.update(streams=17), "streams"),
    (lambda c: c["layers"][0]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][0]["mixer"].update(heads=5), "kv_heads"),
    (lambda c: c["layers"][0].update(type="lightning"), "type"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=14), "rot.dims"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "top"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.9]), "decay"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.9, 1.5]), "decay"),
    (lambda c: c["layers"][2]["mixer"].update(conv=9), "conv"),
    (lambda c: c["layers"][2]["mixer"].update(dim=300), "dim"),
    (lambda c: c["layers"][2]["mixer"]["q_temp"].update(every=0), "every"),
    (lambda c: c["layers"][2]["mlp"].update(kind="sparse"), "kind"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_config_errors_name_the_key(change, word):
    raw = json.loads(json.dumps(fo.FO_A))
    change(raw)
    with pytest.raises(ConfigError) as e:
        api.load_config(raw)
    assert word in str(e.value)


def test_weights_bind_by_name_and_faults_are_listed_together():
    cfg = api.load_config(json.loads(json.dumps(fo.FO_A)))
    arch = registry.find("Fovosun")
    t = fo.draw_tensors(fo.FO_A, 1)
    assert t["l0.mix.q"].shape == (96, 64) and t["l0.mix.k.b"].shape == (48,) and t["l0.mix.v"].shape == (32, 64)
    assert "l0.mix.g" not in t and "l0.mix.q.conv" not in t and "l2.mix.q.b" not in t and "l1.hc2.in" not in t and "l1.norm2" not in t
    assert t["l2.mix.q.conv"].shape == (96, 4) and t["l2.mix.g"].shape == (6, 64) and t["l2.mix.lk2"].shape == (8,)
    assert t["l1.mix.g"].shape == (24, 64) and t["l0.hc2.mix"].shape == (2, 2) and t["l0.mlp.router.b"].shape == (5,)
    model = arch.build(cfg, WeightStore.from_tensors(t, device="cpu", compute_dtype=torch.float32))
    assert model.head.weight.data_ptr() != model.embedding.table.data_ptr() and model.head.norm.streams.tolist() == [1.0, 1.0]
    m0, m1, m2 = (b.mixer for b in model.layers)
    lam = pl.difference_weight(*(t["l0.mix." + n] for n in ("lq1", "lk1", "lq2", "lk2")), 0.3)
    assert abs(m0.lam - lam) < 1e-12 and abs(m0.lam - 0.3) > 0.05
    assert m0.window == 9 and m0.head_dim == 32 and m0.bias.shape == (176,) and not m0.gated and m0.conv is None
    assert m2.gated and m2.conv.taps == 4 and m2.temperature == (0.7, 5) and m2.bias is None and m2.head_dim == 32
    assert m1.key_scale == 0.25 and m1.norm_heads and m1.norm_weight is None and m1.gate == "silu" and m1.activation is None
    b = model.layers[0]
    assert b.pre_mixer.streams.dtype == b.mix_ffn.mix.dtype == torch.float32 and torch.equal(b.mix_ffn.mix, t["l0.hc2.mix"].float())
    assert b.ffn.score == "softmax_chosen" and b.ffn.shared.limit == 0.6 and b.ffn.limit == 1.3 and model.layers[1].ffn is None
    # what the cache manager is asked for: pages, a memory, pages and a convolution's tail
    needs = model.state_needs()
    assert len(needs) == 3 and needs[0].window == 9 and needs[1].shape == (3, 16, 8)
    assert needs[2].parts[0].window is None and needs[2].parts[1].shape == (3, 96 + 48 + 60)
    c = api.load_config(json.loads(json.dumps(fo.FO_C)))                # one tap: no tail
    one = arch.build(c, WeightStore.from_tensors(fo.draw_tensors(fo.FO_C, 1), device="cpu", compute_dtype=torch.float32))
    assert one.state_needs()[0].n_kv_heads == 1 and one.layers[0].mixer.conv.taps == 1
    # the numbers of a second sublayer that layer 1 does not have may stand in the file; anything else may not
    arch.build(cfg, WeightStore.from_tensors(dict(t, **{"l1.hc2.in": torch.zeros(2), "l1.norm2": torch.zeros(64)}), device="cpu",
                                             compute_dtype=torch.float32))
    with pytest.raises(WeightError) as e:
        arch.build(cfg, WeightStore.from_tensors(dict(t, **{"l1.mlp.up": torch.zeros(4, 64)}), device="cpu", compute_dtype=torch.float32))
    assert e.value.unexpected == ["l1.mlp.up"]
    bad = dict(t)
    del bad["l1.mix.g"]
    with pytest.raises(WeightError) as e:
        arch.build(cfg, WeightStore.from_tensors(bad, device="cpu", compute_dtype=torch.float32))
    assert "l1.mix.g" in e.value.missing
    bad = dict(t, **{"l0.hc1.mix": torch.zeros(3, 2, dtype=torch.bfloat16)})
    with pytest.raises((WeightError, ValueError)) as e:
        arch.build(cfg, WeightStore.from_tensors(bad, device="cpu", compute_dtype=torch.float32))
    assert any(n == "l0.hc1.mix" for n, _, _ in e.value.wrong_shape)


# ---- the plain implementation's mechanisms on inputs whose answers are known -------------------------------------------------

def test_plain_streams_by_hand():
    xs = torch.tensor([[[1.0, 2.0]], [[10.0, 20.0]]], dtype=D64)            # two streams of one row
    assert pl.gather_streams(xs, torch.tensor([0.5, 2.0])).tolist() == [[20.5, 41.0]]
    y = torch.tensor([[100.0, 1000.0]], dtype=D64)
    new = pl.scatter_streams(xs, y, torch.tensor([[1.0, 2.0], [3.0, 4.0]]), torch.tensor([0.0, 1.0]))
    assert new[0].tolist() == [[31.0, 62.0]] and new[1].tolist() == [[142.0, 1084.0]]     # [from, to]


def test_plain_convolution_temperature_and_window_by_hand():
    u = torch.tensor([[1.0, 5.0], [10.0, 6.0], [100.0, 7.0]], dtype=D64)
    y = pl.causal_convolution(u, torch.tensor([[3.0, 2.0, 0.5], [0.0, 1.0, 0.0]]))
    assert y[:, 0].tolist() == [0.5, 5.0 + 2.0, 50.0 + 20.0 + 3.0] and y[:, 1].tolist() == [0.0, 5.0, 6.0]
    f = pl.temperature([0, 1, 2, 3, 6, 7], 0.5, 4)
    want = [1.0, 1.0, 1.0, 1.0 + 0.5 * math.log(2), 1.0 + 0.5 * math.log(2), 1.0 + 0.5 * math.log(3)]
    assert torch.allclose(f, torch.tensor(want, dtype=D64))
    assert pl.window_mask(4, 2).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    assert int(pl.window_mask(5, None).sum()) == 15


def test_plain_rotation_keeps_products_of_equal_distance():
    g = torch.Generator().manual_seed(1)
    q, k = torch.randn(1, 1, 10, generator=g, dtype=D64), torch.randn(1, 1, 10, generator=g, dtype=D64)
    dot = lambda i, j: float((pl.rotate_halves(q, torch.tensor([i]), 50.0, 6) * pl.rotate_halves(k, torch.tensor([j]), 50.0, 6)).sum())
    assert abs(dot(9, 4) - dot(25, 20)) < 1e-12 and abs(dot(9, 4) - dot(9, 5)) > 1e-3
    x = pl.rotate_halves(q, torch.tensor([3]), 50.0, 6)
    assert torch.equal(x[..., 6:], q[..., 6:])
    u, v, a = float(q[0, 0, 1]), float(q[0, 0, 4]), 3 * 50.0 ** (-2 / 6)
    assert abs(float(x[0, 0, 1]) - (u * math.cos(a) - v * math.sin(a))) < 1e-12
    assert abs(float(x[0, 0, 4]) - (v * math.cos(a) + u * math.sin(a))) < 1e-12


def test_plain_difference_by_hand():
    lam = pl.difference_weight(torch.tensor([1.0, 2.0]), torch.tensor([0.5, 0.0]), torch.tensor([0.0, 1.0]), torch.tensor([3.0, -1.0]), 0.25)
    assert abs(lam - (math.exp(0.5) - math.exp(-1.0) + 0.25)) < 1e-12
    a1, a2 = torch.tensor([[[5.0, 1.0]]], dtype=D64), torch.tensor([[[1.0, -1.0]]], dtype=D64)
    o = pl.difference(a1, a2, 2.0, 0.4, 0.0)                               # (3, 3): root mean square 3
    assert torch.allclose(o, torch.full_like(o, 0.6))


def test_plain_maps_share_values_and_read_their_own_queries_and_keys():
    """With lambda at zero the second map does not matter; with map 1's queries at zero the first is the mean of values."""
    cfg = fo.config(12, 20, [fo.layer("attention_2", fo.attention(2, 1, 3, 4, 0.5, diff=0.0))])
    t, g = fo.draw_tensors(cfg, 4), torch.Generator().manual_seed(3)
    h = torch.randn(6, 12, generator=g, dtype=D64)
    m = cfg["layers"][0]["mixer"]
    for n in ("lq1", "lk1", "lq2", "lk2"):
        t["l0.mix." + n].zero_()                                            # lambda = 1 - 1 + 0
    y = pl.attention(h, t, "l0.mix.", m, 1e-6)
    other = dict(t)
    for n in ("q", "k"):
        other["l0.mix." + n] = t["l0.mix." + n].clone()
        other["l0.mix." + n].view(-1, 2, 3, 12)[:, 1] = 1.0
    assert torch.allclose(pl.attention(h, other, "l0.mix.", m, 1e-6), y)
    other["l0.mix.q"] = t["l0.mix.q"].clone()
    other["l0.mix.q"].view(-1, 2, 3, 12)[:, 0] = 0.0
    other["l0.mix.q.b"] = torch.zeros_like(t["l0.mix.q.b"])
    v = h @ t["l0.mix.v"].to(D64).T + t["l0.mix.v.b"].to(D64)
    mean = torch.stack([v[:i + 1].mean(0) for i in range(6)])
    want = torch.cat([pl.rms(mean, 1e-6)] * 2, dim=1) @ t["l0.mix.o"].to(D64).T
    assert torch.allclose(pl.attention(h, other, "l0.mix.", m, 1e-6), want)


def test_plain_decayed_memory_by_hand():
    q, k = torch.ones(3, 1, 1, dtype=D64), torch.tensor([2.0, 1.0, 3.0], dtype=D64).view(3, 1, 1)
    v = torch.tensor([[1.0, -1.0], [4.0, 0.0], [0.0, 2.0]], dtype=D64).view(3, 1, 2)
    assert pl.decayed_memory(q, k, v, [0.5])[:, 0].tolist() == [[2, -2], [5, -1], [2.5, 5.5]]
    assert pl.decayed_memory(q, k, v, [0.0])[2, 0].tolist() == [0, 6] and pl.decayed_memory(q, k, v, [1.0])[2, 0].tolist() == [6, 4]


def test_plain_router_and_clamped_expert_by_hand():
    (row,) = pl.route(torch.tensor([[0.0, 2.0, 1.0, 2.0]], dtype=D64), 3)
    assert [e for e, _ in row] == [1, 3, 2] and abs(row[0][1] - 1 / (2 + math.exp(-1))) < 1e-12 and abs(sum(x for _, x in row) - 1) < 1e-12
    w = {"gate": torch.tensor([[5.0], [-3.0]]), "up": torch.tensor([[-4.0], [0.5]]), "down": torch.tensor([[1.0, 10.0]])}
    y = float(pl.clamped_feed_forward(torch.ones(1, 1, dtype=D64), w, "", 2.0))
    s = lambda z: 1 / (1 + math.exp(-1.702 * z))
    assert abs(y - (2 * s(2) * (-2 + 1) + 10 * (-3 * s(-3) * 1.5))) < 1e-12            # only the gate's lower side is open


# ---- the engine's host logic ------------------------------------------------------------------------------------------

@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
@pytest.mark.parametrize("mode", ["whole", "chunks", "mixed"])
def test_host_logic_on_the_cpu_stand_in(name, mode, tmp_path, cpu_ops):
    cfg, lengths, page = fo.CASES[name]
    folder = fo.write_model(str(tmp_path / "m"), cfg, seed=3)
    reqs = {f"r{i}": helpers.random_tokens(n, cfg["vocab"], 100 + i) for i, n in enumerate(lengths)}
    tensors = helpers.read_tensors(folder)
    ref = {rid: pl.forward(cfg, tensors, toks).float() for rid, toks in reqs.items()}
    steps = {"whole": helpers.trace_whole, "chunks": helpers.trace_chunks, "mixed": lambda r: helpers.trace_mixed(r, seed=4)}[mode](reqs)
    runner = _runner(folder, page, helpers.trace_max_tokens(steps, page))
    got = helpers.run_trace_with_runner(runner, steps)
    assert len(got) == sum(lengths)
    assert _rel(got, ref) < 3e-4
    assert runner.cache.n_live == 0
    runner.cache.check()


def test_a_window_gives_its_pages_back_beside_a_layer_without_one(cpu_ops, tmp_path):
    from kungfu_b200.engine import StepEntry
    cfg = fo.config(32, 60, [fo.layer("attention_2", fo.attention(2, 1, 4, 8, 0.6, window=6, rot=(50.0, 4))),
                             fo.layer("attention", fo.attention(2, 2, 4, 6, 0.6, conv=3, temp=(0.5, 4)))], streams=2)
    folder = fo.write_model(str(tmp_path / "m"), cfg, seed=5)
    toks = helpers.random_tokens(41, 60, 3)
    ref = pl.forward(cfg, helpers.read_tensors(folder), toks).float()
    runner = _runner(folder, 4, 64, max_requests=1)
    assert [g.window for g in runner.cache.groups] == [6, None]
    runner.cache.add_request("a")
    got, at = {}, 0
    for n in (9, 1, 2, 7, 1, 12, 7, 1, 1):
        out = runner.step([StepEntry("a", toks[at:at + n], list(range(n)))])
        for i in range(n):
            got[("a", at + i)] = out[i].clone()
        at += n
    held = [[i for i, p in enumerate(runner.cache.block_table(g, "a")) if p >= 0] for g in (0, 1)]
    assert at == 41 and _rel(got, {"a": ref}) < 3e-4 and held == [[9, 10], list(range(11))]
    runner.cache.release("a")
    runner.cache.check()


def _greedy_is_plain(cfg, tensors, prompts, outs, n):
    for p, o in zip(prompts, outs):
        assert len(o) == n
        seq = list(p)
        for tok in o:
            logits = pl.forward(cfg, tensors, seq)[-1]
            top = torch.topk(logits, 2).values
            if float(top[0] - top[1]) > 1e-3 * float(logits.abs().max()):
                assert int(torch.argmax(logits)) == tok
            seq.append(tok)


def test_greedy_generation_through_the_scheduler(cpu_ops, tmp_path):
    """Portions under a token budget beside decode rows, through the engine's scheduler, against the plain
    implementation's best token at every place; also with a pool so small that a request is sent back and starts anew
    (its memory and its convolution tails start from nothing again)."""
    from kungfu_b200.engine.engine import Engine
    from kungfu_b200.sampling import Sampling
    cfg = fo.config(48, 150, [fo.layer("attention", fo.attention(2, 1, 8, 12, 0.4, conv=3, temp=(0.5, 6)), fo.dense(40)),
                              fo.layer("retention", fo.retention(2, 8, 12, [0.9, 0.99], rot=(100.0, 8)), fo.moe(4, 2, 20, shared=(12, 1.0))),
                              fo.layer("attention_2", fo.attention(2, 2, 6, 8, 0.4, window=6, rot=(100.0, 6)))])
    folder = fo.write_model(str(tmp_path / "m"), cfg, seed=9)
    tensors = helpers.read_tensors(folder)

    def engine(pool, batch):
        c, model = api.load_model(folder, dtype="float32", device="cpu")
        runner = api.make_runner(c, model, dtype="float32", device="cpu", page_size=4, max_tokens=pool, max_requests=4, max_context=96)
        return Engine(runner=runner, batch=batch, parallel=4)

    prompts = [helpers.random_tokens(n, cfg["vocab"], 40 + n) for n in (19, 2, 31, 8)]
    eng = engine(512, 8)
    _greedy_is_plain(cfg, tensors, prompts, eng.generate(prompts, Sampling(temperature=0.0), max_tokens=8, ignore_eos=True), 8)
    assert eng.scheduler.n_preemptions == 0
    short = [helpers.random_tokens(n, cfg["vocab"], 90 + n) for n in (5, 7, 6)]
    tight = engine(36, 16)
    _greedy_is_plain(cfg, tensors, short, tight.generate(short, Sampling(temperature=0.0), max_tokens=8, ignore_eos=True), 8)
    assert tight.scheduler.n_preemptions > 0 and tight.runner.cache.n_live == 0
