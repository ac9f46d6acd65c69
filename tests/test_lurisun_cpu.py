"""Lurisun without a GPU: configuration and weights, the plain implementation's own mechanisms on hand-made inputs, and
the engine's host logic (pages of windows and chunks, state slots of memories, convolution tails and the token before,
portions, mixed batches) with the kernels replaced by the CPU stand-in, against the plain implementation."""
import json
import math

import pytest
import torch

import helpers
import lurisun_cases as lu
import plain_lurisun as pl
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
    cfg = api.load_config(json.loads(json.dumps(lu.LU_A)))
    assert (cfg.architecture, cfg.width, cfg.vocab, len(cfg.layers)) == ("Lurisun", 64, 300, 3)
    assert (cfg.norm_eps, cfg.logit_scale, cfg.taps) == (1e-6, 3.5, 4)
    assert (cfg.pair.mul_prev, cfg.pair.mul_cur, cfg.pair.buckets) == (7, 3, 61)
    a, l, c = (x.mixer for x in cfg.layers)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.chunk, a.rot_base, a.rot_dims) == (4, 2, 24, 24, 0.2, 9, 100.0, 8)
    assert (l.heads, l.dim, l.vdim, l.decay) == (3, 16, 8, (0.5, 0.9, 0.995))
    assert (c.heads, c.dim, c.vdim, c.kv_rank, c.q_rank, c.scale, c.window) == (3, 8, 12, 20, 28, 0.4, 7)
    assert [x.ff for x in cfg.layers] == [72, 0, 40]
    for case in (lu.LU_A, lu.LU_B, lu.LU_C, lu.LU_D, lu.LU_E):
        one = api.load_config(json.loads(json.dumps(case)))
        assert api.load_config(json.loads(json.dumps(one.to_dict()))) == one
    c = api.load_config(json.loads(json.dumps(lu.LU_C)))
    assert c.layers[3].mixer.chunk is None and c.layers[1].mixer.rot_dims == 0 and c.logit_scale == 1.0
    rows = cfg.state_summary()
    assert [r["kind"] for r in rows] == ["kv_pages", "memory", "latent_pages"]
    assert rows[1]["fixed_bytes"] == 4 * (3 * 64 + 3 * 16 * 8) and rows[0]["window"] == 9 and rows[2]["window"] == 7


@pytest.mark.parametrize("change,word", [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c.pop("canon"), "canon"),
    (lambda c: c["canon"].update(taps=9), "taps"),
    (lambda c: c["embedding"]["bigram"].pop("buckets"), "buckets"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=8), "vdim"),
    (lambda c: c["layers"][0].update(type="delta"), "type"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.9]), "decay"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.9, 1.5]), "decay"),
    (lambda c: c["layers"][2]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][2]["mlp"].update(kind="moe"), "kind"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_config_errors_name_the_key(change, word):
    raw = json.loads(json.dumps(lu.LU_A))
    change(raw)
    with pytest.raises(ConfigError) as e:
        api.load_config(raw)
    assert word in str(e.value)


def test_weights_bind_by_name_and_faults_are_listed_together():
    cfg = api.load_config(json.loads(json.dumps(lu.LU_A)))
    arch = registry.find("Lurisun")
    t = lu.draw_tensors(lu.LU_A, 1)
    assert t["bigram"].shape == (62, 64) and t["l0.mix.k"].shape == (48, 64) and "l0.mix.v" not in t and t["l0.mix.pb"].shape == (4,)
    assert t["l0.mix.q.norm"].shape == (96,) and t["l1.mix.norm"].shape == (24,) and "l1.norm2" not in t and t["l1.canon1"].shape == (64, 4)
    assert t["l2.mix.uq"].shape == (24, 28) and t["l2.mix.g"].shape == (36, 64) and t["head"].shape == (300, 64)
    model = arch.build(cfg, WeightStore.from_tensors(t, device="cpu", compute_dtype=torch.float32))
    assert model.head.weight.data_ptr() != model.embedding.table.data_ptr()
    assert torch.allclose(model.head.norm.weight, 3.5 * t["final.norm"].float())
    m0, m1, m2 = (b.mixer for b in model.layers)
    assert m0.values_are_keys and m0.chunk == 9 and m0.window is None and m0.sigmoid_bias.dtype == torch.float32
    assert m0.w_in.shape[0] == 96 + 48 and not m0.position.interleaved and m0.position.rotary_dims == 8
    assert m1.powers.shape[0] == 3 and torch.allclose(m1.powers[:, 2], torch.tensor([0.25, 0.81, 0.995 ** 2]))
    assert m2.gate_elements and m2.window == 7 and m2.head_dim == 32
    # what the cache manager is asked for: pages or a memory, each with the convolution's tail; last, the token before
    needs = model.state_needs()
    assert len(needs) == 4 and needs[0].parts[0].chunk == 9 and needs[0].parts[1].shape == (3, 64)
    assert needs[1].parts[0].shape == (3, 16, 8) and needs[2].parts[0].window == 7
    assert needs[3].shape == (1,) and needs[3].dtype == torch.int32
    d = api.load_config(json.loads(json.dumps(lu.LU_D)))                # one tap: no tail
    one = arch.build(d, WeightStore.from_tensors(lu.draw_tensors(lu.LU_D, 1), device="cpu", compute_dtype=torch.float32))
    assert one.state_needs()[0].shape == (1, 4, 6)
    bad = dict(t)
    del bad["l1.mix.norm"]
    bad["l0.mix.pb"] = torch.zeros(5, dtype=torch.bfloat16)
    with pytest.raises(WeightError) as e:
        arch.build(cfg, WeightStore.from_tensors(bad, device="cpu", compute_dtype=torch.float32))
    assert any(n == "l0.mix.pb" for n, _, _ in e.value.wrong_shape)


# ---- the plain implementation's mechanisms on inputs whose answers are known -------------------------------------------------

def test_plain_pair_rows_by_hand():
    assert pl.bigram_rows([5, 2, 9], 7, 3, 11) == [11, (35 + 6) % 11, (14 + 27) % 11]
    assert pl.bigram_rows([4], 1, 1, 3) == [3]
    w = {"embed": torch.eye(4), "bigram": torch.diag(torch.tensor([10.0, 20.0, 30.0]))[:, :3]}
    w["bigram"] = torch.cat([w["bigram"], torch.zeros(3, 1)], dim=1)
    x = pl.embedding([3, 1], w, {"embedding": {"bigram": {"mul_prev": 1, "mul_cur": 2, "buckets": 2}}})
    assert x[0].tolist() == [0, 0, 30, 1] and x[1].tolist() == [0, 1 + 20, 0, 0]           # (3 + 2) mod 2 = 1


def test_plain_input_convolution_by_hand():
    h = torch.tensor([[1.0], [10.0], [100.0]], dtype=D64)
    y = pl.input_convolution(h, torch.tensor([[3.0, 2.0, 0.5]]))
    assert y[:, 0].tolist() == [1.5, 15.0 + 2.0, 150.0 + 20.0 + 3.0]


def test_plain_decayed_memory_by_hand():
    q, k = torch.ones(3, 1, 1, dtype=D64), torch.tensor([2.0, 1.0, 3.0], dtype=D64).view(3, 1, 1)
    v = torch.tensor([[1.0, -1.0], [4.0, 0.0], [0.0, 2.0]], dtype=D64).view(3, 1, 2)
    o = pl.decayed_memory(q, k, v, [0.5])
    assert o[:, 0].tolist() == [[2, -2], [5, -1], [2.5, 5.5]]                             # the token itself is already in
    assert pl.decayed_memory(q, k, v, [0.0])[2, 0].tolist() == [0, 6]
    assert pl.decayed_memory(q, k, v, [1.0])[2, 0].tolist() == [6, 4]


def test_plain_masks_by_hand():
    c = pl.chunk_mask(7, 3)
    assert c[5].tolist() == [False, False, False, True, True, True, False] and c[3].tolist() == [False] * 3 + [True] + [False] * 3
    assert c[2].tolist() == [True, True, True] + [False] * 4
    m = pl.window_mask(7, 3)
    assert m[5].tolist() == [False, False, False, True, True, True, False] and m[3].tolist() == [False, True, True, True] + [False] * 3
    assert pl.chunk_mask(4, None)[3].tolist() == [True] * 4 and pl.window_mask(4, 1).tolist() == torch.eye(4, dtype=torch.bool).tolist()


def test_plain_sigmoid_attention_by_hand():
    q, k = torch.full((2, 1, 1), math.log(3.0), dtype=D64), torch.ones(2, 1, 1, dtype=D64)
    v = torch.tensor([2.0, -4.0], dtype=D64).view(2, 1, 1)
    o = pl.sigmoid_attend(q, k, v, 1.0, torch.zeros(1), pl.chunk_mask(2, None))
    assert float(o[0]) == pytest.approx(0.75 * 2.0) and float(o[1]) == pytest.approx(0.75 * (2.0 - 4.0))       # not normalized
    o = pl.sigmoid_attend(q, k, v, 2.0, torch.tensor([-2 * math.log(3.0)]), pl.chunk_mask(2, 1))
    assert float(o[0]) == pytest.approx(0.5 * 2.0) and float(o[1]) == pytest.approx(0.5 * -4.0)


def test_plain_rotation_pairs_by_hand():
    x = torch.zeros(3, 1, 10, dtype=D64)
    x[:, 0, 0], x[:, 0, 9] = 1.0, 7.0
    pos, ang = torch.tensor([0, 1, 5]), torch.tensor([0.0, 1.0, 5.0], dtype=D64)
    y = pl.rotate_halves(x, pos, 100.0, 8)
    assert torch.allclose(y[:, 0, 0], torch.cos(ang)) and torch.allclose(y[:, 0, 4], torch.sin(ang))
    assert float((y[:, 0, 9] - 7.0).abs().max()) == 0.0 and float(y[:, 0, 8].abs().max()) == 0.0
    x = torch.zeros(1, 1, 8, dtype=D64)
    x[0, 0, 7] = 1.0                                       # the second of the last pair, which turns slowest
    y = pl.rotate_halves(x, torch.tensor([4]), 16.0, 8)
    assert float(y[0, 0, 3]) == pytest.approx(-math.sin(4 * 16.0 ** -0.75)) and float(y[0, 0, 7]) == pytest.approx(math.cos(0.5))


def test_plain_attention_takes_the_keys_as_projected_for_values():
    g = torch.Generator().manual_seed(5)
    W, H, G, d, T = 12, 4, 2, 6, 9
    w = {"p.q": torch.randn(H * d, W, generator=g), "p.k": torch.randn(G * d, W, generator=g), "p.q.b": torch.randn(H * d, generator=g),
         "p.k.b": torch.randn(G * d, generator=g), "p.q.norm": torch.rand(H * d, generator=g), "p.k.norm": torch.rand(G * d, generator=g),
         "p.pb": torch.full((H,), 50.0), "p.o": torch.eye(H * d)}
    h = torch.randn(T, W, generator=g, dtype=D64)
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": 0.1, "mask": {"size": 1}, "rot": {"base": 10.0, "dims": 4}}
    y = pl.attention(h, w, "p.", m, 1e-6)                  # chunks of one, weights of one: the token's own value
    k = h @ w["p.k"].to(D64).T + w["p.k.b"].to(D64)        # biased, neither normed nor turned
    assert torch.allclose(y, k.view(T, G, 1, d).expand(T, G, 2, d).reshape(T, H * d))


def test_plain_latent_space_form_is_the_same_attention():
    """Queries taken into the latent space and the values' map applied after the weighted sum: the same numbers."""
    cfg = lu.config(32, 50, [lu.layer("latent_attention", lu.latent(3, 6, 5, 9, 7, 0.5, window=4))])
    t = lu.draw_tensors(cfg, 6)
    h = torch.randn(11, 32, generator=torch.Generator().manual_seed(2), dtype=D64)
    m = cfg["layers"][0]["mixer"]
    plain = pl.latent_attention(h, t, "l0.mix.", m, 1e-6)
    saved = pl.ROUND
    pl.ROUND = lambda x: x * 1.0                               # not the marker of exact arithmetic, and yet exact
    try:
        other = pl.latent_attention(h, t, "l0.mix.", m, 1e-6)
    finally:
        pl.ROUND = saved
    assert torch.allclose(plain, other, atol=1e-12)


# ---- the engine's host logic ------------------------------------------------------------------------------------------

@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
@pytest.mark.parametrize("mode", ["whole", "chunks", "mixed"])
def test_host_logic_on_the_cpu_stand_in(name, mode, tmp_path, cpu_ops):
    cfg, lengths, page = lu.CASES[name]
    folder = lu.write_model(str(tmp_path / "m"), cfg, seed=3)
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


def test_pages_of_finished_chunks_go_back(cpu_ops, tmp_path):
    """A layer of chunks gives back every page of the chunks before the next token's, as soon as that token would start
    a new chunk; one that shares a page with the next chunk stays."""
    from kungfu_b200.engine import StepEntry
    cfg = lu.config(32, 60, [lu.layer("attention", lu.attention(2, 1, 8, 0.4, chunk=10, rot_dims=4, base=50.0))], taps=2)
    folder = lu.write_model(str(tmp_path / "m"), cfg, seed=5)
    toks = helpers.random_tokens(43, 60, 3)
    ref = pl.forward(cfg, helpers.read_tensors(folder), toks).float()
    runner = _runner(folder, 4, 64, max_requests=1)
    runner.cache.add_request("a")
    got, at = {}, 0
    held = {}
    for n in (9, 1, 2, 7, 1, 3, 7, 9, 2, 1, 1):
        out = runner.step([StepEntry("a", toks[at:at + n], list(range(n)))])
        for i in range(n):
            got[("a", at + i)] = out[i].clone()
        at += n
        held[at] = [i for i, p in enumerate(runner.cache.block_table(0, "a")) if p >= 0]
    assert at == 43 and _rel(got, {"a": ref}) < 3e-4
    # length 9: token 9 still reads from token 0; length 10: token 10 starts a chunk, whose first page (tokens 8..11) stays
    assert held[9] == [0, 1, 2] and held[10] == [2] and held[12] == [2]
    assert held[19] == [2, 3, 4] and held[20] == [] and held[39] == [7, 8, 9] and held[41] == [10] and held[43] == [10]
    from kungfu_b200.cache.kinds import lifetime_chunked, lifetime_keep, lifetime_name, lifetime_window
    key = runner.cache.groups[0].window
    assert lifetime_chunked(key) and lifetime_window(key) == 10 and lifetime_keep(key) == 0 and lifetime_name(key) == "chunk10"
    assert [lifetime_name(k) for k in (None, 7, (7, 2))] == ["none", "7", "7+2"]
    runner.cache.release("a")
    runner.cache.check()


def test_windows_and_chunks_of_one_size_are_groups_of_their_own(cpu_ops, tmp_path):
    cfg = lu.config(32, 60, [lu.layer("attention", lu.attention(2, 1, 8, 0.4, chunk=8)), lu.layer("latent_attention", lu.latent(2, 4, 4, 8, 8, 0.4, window=8)),
                             lu.layer("attention", lu.attention(1, 1, 8, 0.4)), lu.layer("attention", lu.attention(4, 2, 4, 0.4, chunk=8))], taps=3)
    folder = lu.write_model(str(tmp_path / "m"), cfg, seed=5)
    runner = _runner(folder, 4, 64)
    assert [g.window for g in runner.cache.groups] == [("chunk", 8), 8, None] and runner.cache.groups[0].slots == [0, 3]
    toks = helpers.random_tokens(30, 60, 3)
    ref = pl.forward(cfg, helpers.read_tensors(folder), toks).float()
    got = helpers.run_trace_with_runner(runner, helpers.trace_chunks({"a": toks}))
    assert _rel(got, {"a": ref}) < 3e-4


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
    (its memory, its convolution tails and the token before start from nothing again)."""
    from kungfu_b200.engine.engine import Engine
    from kungfu_b200.sampling import Sampling
    cfg = lu.config(48, 150, [lu.layer("attention", lu.attention(2, 1, 8, 0.4, rot_dims=4), 40),
                              lu.layer("lightning", lu.lightning(2, 8, 12, [0.9, 0.99]), 30),
                              lu.layer("latent_attention", lu.latent(2, 8, 6, 12, 10, 0.3, window=6), 30)], taps=3, logit_scale=2.0)
    folder = lu.write_model(str(tmp_path / "m"), cfg, seed=9)
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
